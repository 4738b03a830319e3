// Decoder designs the native loop serves besides the litnicelm transformer: a
// model folder (config.json + model.safetensors) names its architecture, the
// registry (model_registry.cu) makes the matching DecoderModel, and the session
// drives it with its own loop, sampler, graphs and slots.
#pragma once

#include <memory>
#include <string>
#include <vector>

#include "common.cuh"
#include "json.hpp"

namespace lb {

// How a model computes: BF16 = bfloat16 weights and matrix-product operands with
// 32-bit accumulation (norms, attention scores and weights, the residual stream
// and recurrent state stay 32-bit); F32 = everything in 32-bit.
enum class Precision : int { BF16 = 0, F32 = 1 };

// The tensors of a safetensors file (8-byte little-endian header length, JSON
// header name -> {dtype, shape, data_offsets}, data).
class TensorFile {
 public:
  struct Entry {
    std::string name, dtype;
    std::vector<long long> shape;
    uint64_t begin = 0, end = 0;  // bytes inside the data section
  };
  explicit TensorFile(const std::string &path);
  const std::string &path() const { return path_; }
  uint64_t data_offset() const { return data_offset_; }
  uint64_t data_bytes() const { return data_bytes_; }
  bool has(const std::string &name) const { return lookup(name) != nullptr; }
  // The entry, checked: bfloat16 and exactly this shape.
  const Entry &bf16(const std::string &name, const std::vector<long long> &shape) const;
  // The shape of a tensor (the entry must exist).
  const std::vector<long long> &shape(const std::string &name) const;
  // One bfloat16 number (shape [] or [1]), read on the host.
  float scalar_bf16(const std::string &name) const;

 private:
  const Entry *lookup(const std::string &name) const;
  std::string path_;
  uint64_t data_offset_ = 0, data_bytes_ = 0;
  std::vector<Entry> entries_;
};

// The new rows of one step: positions p0 .. p0 + n - 1 of the streams in slots
// slot0 .. slot0 + streams - 1 (row r = stream * n + t). Their token ids lie at
// ids[slot * ids_ld + position]. state != nullptr (graph replay, n == 1): the
// position is state->s - 1 and s_cap bounds the context length state->s.
struct RowBatch {
  int streams = 1, slot0 = 0;
  int p0 = 0, n = 1;
  int s_cap = 0;
  const LoopState *state = nullptr;
  const int *ids = nullptr;
  int ids_ld = 0;
  long long rows() const { return (long long)streams * n; }
};

class DecoderModel {
 public:
  virtual ~DecoderModel() = default;
  virtual const char *architecture() const = 0;
  virtual int n_layers() const = 0;
  virtual int width() const = 0;
  virtual int vocab() const = 0;
  // Positions the design has vectors for; 0: no bound of its own.
  virtual int max_positions() const = 0;
  virtual void load(const TensorFile &file, cudaStream_t st, DevErr *err) = 0;
  // Room for `streams` slots of `cap` positions each (what the slots hold is kept) and for steps of
  // `rows` new rows. Returns true when a buffer that a captured graph may point at has moved.
  virtual bool reserve(int streams, int cap, long long rows, cudaStream_t st) = 0;
  // The forward pass of the new rows through every layer; the slots' state is advanced. Returns the
  // number of kernels launched.
  virtual int enqueue_rows(const RowBatch &batch, cudaStream_t st, DevErr *err) = 0;
  // Logits [n_rows, vocab] of rows of the batch just enqueued: the rows listed at rows_dev (device
  // memory), or, with rows_dev == nullptr, the last row of every stream. logits has room for n_rows
  // rounded up to a multiple of 8.
  virtual int enqueue_head(const RowBatch &batch, const int *rows_dev, int n_rows, float *logits, cudaStream_t st,
                           DevErr *err) = 0;
  // Contexts of one bucket replay the same captured step: its upper bound for a context of s.
  virtual int context_bound(int s) const = 0;
  // New rows a step should bring at most (longer prompts are cut into portions).
  virtual long long portion_rows() const = 0;
};

// model_registry.cu
std::unique_ptr<DecoderModel> make_model(const Json &config, Precision precision);
const char *registered_architectures();  // names with commas between them
std::string read_text_file(const std::string &path);

// ---- kernels of these designs ------------------------------------------------
// Inside these kernels only weights are __restrict__ const: such loads count as invariant and may be
// scheduled ahead of the wait for the preceding kernel (pdl_wait), which wrote every other input.

// embed.cu: x[r, :] = table[ids] * scale + pos[p] for the rows of a batch (pos may be null); tables bfloat16 or float.
void launch_embed_rows(const void *table, const void *pos, float scale, Precision type, const RowBatch &b, int d, int vocab, float *x,
                       cudaStream_t st, DevErr *err);

// canon.cu: h = x / sqrt(mean(x^2) + eps) * gain (one gain for all coordinates), then for each of up
// to two sublayers a_i = h + conv_i(h), a causal convolution over time per channel with `taps` taps.
// history: [slots][taps - 1][d] float, the last inputs h of every slot at position % (taps - 1).
struct CanonConv {
  const float *w = nullptr;  // [taps][d]
  void *out = nullptr;       // [rows, ld], bfloat16 or float by Precision
  int ld = 0;
};
void launch_rms_canon(const float *x, int d, float gain, float eps, int taps, float *history, const CanonConv *conv,
                      int n_conv, Precision type, const RowBatch &b, cudaStream_t st);
// Gain of an RMS norm: base + w[c], or base alone for all coordinates. Weights stored around zero take base 1.
struct RmsWeight {
  const float *w = nullptr;
  float base = 0.f;
  __device__ __forceinline__ float at(int c) const { return w ? base + w[c] : base; }
};
// canon.cu: RMS norm of listed rows (rows_dev) or of every stream's last row.
void launch_rms_rows(const float *x, int d, const RmsWeight &weight, float eps, const int *rows_dev, int n_rows, int n_per_stream,
                     void *out, int ld, Precision type, cudaStream_t st);

// latent_attention.cu. A latent cache is [slots][cap][ld] (bfloat16 or float): one compressed row per
// position, from which every head's key and value are linear maps.
struct LatentCache {
  void *rows = nullptr;
  int cap = 0, ld = 0, rank = 0;
};
// New rows' latents c = rms(dkv) * gain into the cache (dkv != nullptr), and, with packed != nullptr, the
// rows of positions first .. p0 + n - 1 of every stream side by side: packed[stream * packed_rows + (p - first)].
void launch_latent_store(const float *dkv, int dkv_ld, const float *gain, float eps, const LatentCache &cache,
                         void *packed, int packed_rows, int first, Precision type, const RowBatch &b, cudaStream_t st);

// Sliding-window latent attention: head h of the row at position p attends to positions j with
// 0 <= p - j < window through scores scale * q_h . (W_uk c_j)_h and sums W_uv c_j.
struct LatentAttention {
  int heads, dim, vdim;
  float scale;
  int window;
  const void *q;        // [rows, q_ld]: heads side by side, dim each (bfloat16 or float)
  int q_ld;
  const void *w_uk;     // [heads * dim, w_ld]
  const void *w_uv;     // [heads * vdim, w_ld]
  int w_ld;
  LatentCache cache;
  void *out;            // [rows, out_ld]: heads side by side, vdim each
  int out_ld;
};
// Any size, 32-bit arithmetic on CUDA cores, one CTA per row and head.
void launch_latent_attention_rows(const LatentAttention &a, Precision type, const RowBatch &b, cudaStream_t st);
// Few new rows (decoding and short portions) on bfloat16: W_uk absorbed into the query, key chunks
// shared by 16 heads, partial results joined and mapped through W_uv. fresh: the rows' W_dkv h, stored
// into the cache on the way (dkv == nullptr: the layer reads latents another layer has stored). Returns
// the kernels launched.
struct LatentFresh {
  const float *dkv = nullptr;  // [rows, ld]
  int ld = 0;
  const float *gain = nullptr;
  float eps = 0.f;
};
bool latent_decode_supports(const LatentAttention &a);
size_t latent_decode_scratch_floats(int heads, int rank, int window, int s_cap, long long rows);
int launch_latent_decode(const LatentAttention &a, const LatentFresh &fresh, float *scratch, const RowBatch &b,
                         cudaStream_t st);

// prefill_attention_tc.cu: many new rows on bfloat16 tensor cores over expanded keys and values:
// k [streams * key_rows, k_ld] row-major, vt [heads * vdim, vt_ld] with one column per key; key row j
// of a stream is position first + j.
bool latent_prefill_supports(int dim, int vdim);
void launch_latent_prefill(const LatentAttention &a, const void *k, int k_ld, const void *vt, int vt_ld, int key_rows,
                           int first, const RowBatch &b, cudaStream_t st, DevErr *err);

// residual_norm.cu: the norms around a sublayer in one pass over the residual stream x [rows, d]:
//   x <- x + rms(y) * after      (y == nullptr: x stays)
//   h  = rms(x) * before         (h == nullptr: not asked for)
// y [rows, d] float, h [rows, h_ld] bfloat16 or float.
void launch_residual_norm(float *x, const float *y, const RmsWeight &after, void *h, int h_ld, const RmsWeight &before, int d,
                          long long rows, float eps, Precision type, cudaStream_t st);

// Which keys a query at position p sees besides j <= p: the last `size` positions, or those of its own chunk of
// `size` positions counted from 0.
enum class SpanKind : int { WINDOW = 0, CHUNK = 1 };
struct KeySpan {
  SpanKind kind = SpanKind::WINDOW;
  int size = 1;
  // First key of the query at p (may be negative for a window).
  __host__ __device__ __forceinline__ int first(int p) const {
    return kind == SpanKind::CHUNK ? p - p % size : p - size + 1;
  }
};

// Rotary positions: dimension i of a head turns together with i + dims / 2 by p * turns[i] half turns (turns: angle
// per position over pi, double), both results times `amplitude`; dimensions from dims on pass.
struct Rotation {
  int dims = 0;
  const double *turns = nullptr;  // [dims / 2], device
  float amplitude = 1.f;
};

// grouped_attention.cu: softmax attention whose query heads share key and value heads. Heads are padded to
// multiples of 16 elements with zeros everywhere (dim, vdim: padded sizes); caches are [slots][cap][groups * dim] and
// [slots][cap][groups * vdim].
struct GroupedAttention {
  int heads, groups, dim, vdim;
  float scale;
  KeySpan span;
  const void *q;   // [rows, q_ld]
  int q_ld;
  void *k_cache, *v_cache;
  int cap, slots;
  void *out;       // [rows, out_ld], heads side by side, vdim each
  int out_ld;
};
// Queries and keys: RMS norm over all heads of a row at once (weights [heads * dim] and [groups * dim], true_dim of each
// dim counted), rotation, queries to q, keys and values to the caches. src rows: [queries | keys | values], ld apart.
void launch_qk_norm_rotate(const void *src, int ld, const float *q_weight, const float *k_weight, float eps, int true_dim,
                           const Rotation &rot, const GroupedAttention &a, void *q, Precision type, const RowBatch &b,
                           cudaStream_t st);
// Any number of rows, 32-bit arithmetic on CUDA cores; keys split over a cluster's CTAs where rows are few.
void launch_grouped_attention_rows(const GroupedAttention &a, Precision type, const RowBatch &b, cudaStream_t st);
// prefill_attention_tc.cu: many new rows on bfloat16 tensor cores, keys and values as they lie in the caches.
bool grouped_prefill_supports(int dim, int vdim);
void launch_grouped_prefill(const GroupedAttention &a, const RowBatch &b, cudaStream_t st, DevErr *err);

// delta.cu, delta_chunk.cu: the gated delta rule. Per head, with unit vectors q, k and the state S [dim, vdim]:
//   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// after a short causal convolution and SiLU on q, k and v; o is normalised per head and gated. dim and vdim are
// padded to multiples of 16 with zeros. Columns of a projected row: [q | k | v | gate], groups * dim twice and
// heads * vdim twice, and beside them [beta | decay] in float.
struct DeltaMixer {
  int heads, groups, dim, vdim;   // padded sizes
  int true_dim, true_vdim;        // q scale, and what the output's norm counts
  int taps;
  float eps;
  const float *conv;              // [taps][conv_channels]
  const float *a_log, *dt_bias;   // [heads]
  const float *norm;              // [vdim]
  float *state;                   // [slots][heads][dim][vdim]
  void *history;                  // [slots][taps][conv_channels]: inputs of the convolution, position % taps
  const void *in;                 // [rows, in_ld] bfloat16 or float
  int in_ld;
  const float *ba;                // [rows, ba_ld]
  int ba_ld;
  void *out;                      // [rows, out_ld]
  int out_ld;
  int conv_channels() const { return 2 * groups * dim + heads * vdim; }
};
// What launch_delta needs besides: convolved rows [rows][conv_channels], outputs before the norm
// [rows][heads * vdim] float, and the chunked form's matrices.
size_t delta_scratch_bytes(const DeltaMixer &m, long long rows, int streams, Precision type);
// The new rows' recurrence and gated norm, state and history advanced; returns the kernels launched.
int launch_delta(const DeltaMixer &m, void *scratch, Precision type, const RowBatch &b, cudaStream_t st, DevErr *err);
bool delta_supports(int dim, int vdim);

// Activations of the products and of launch_activation_f32: GELU in its error-function and tanh forms.
enum Activation : int { ACT_NONE = 0, ACT_GELU_ERF = 1, ACT_GELU_TANH = 2 };

// Matrix products on bfloat16 with 32-bit accumulation: C[m, n] = A[m, k] W[n, k]^T.
struct Bf16Product {
  const void *a = nullptr;  // [rows, a_ld] bfloat16; a_ld % 8 == 0
  int a_ld = 0;
  const void *w = nullptr;  // [n, w_ld] bfloat16; w_ld % 8 == 0
  int w_ld = 0;
  int n = 0, k = 0;
  // result: columns below n_half go to half_out (bfloat16, through the activation), the others to
  // float_out[:, column - n_half] (added to what it holds when accumulate is set)
  int n_half = 0;
  void *half_out = nullptr;
  int half_ld = 0;
  int act = ACT_NONE;
  // gated: columns 2 j and 2 j + 1 below n_half are a gate and its factor, half_out[:, j] = act(c_2j) * c_2j+1
  int gated = 0;
  float *float_out = nullptr;
  int float_ld = 0;
  int accumulate = 0;
};
// few_row_bf16.cu: m <= 64 rows, bound by the weights' bytes; up to two products in one launch.
constexpr int FEW_ROWS_MAX = 64;
void launch_few_row_bf16(const Bf16Product *p, int count, int m, cudaStream_t st);
// gemm_bf16.cu: any m, on the tensor cores (tcgen05).
void launch_gemm_bf16(const Bf16Product &p, int m, cudaStream_t st, DevErr *err);

// weights.cu: tensors of a file image in device memory to the layouts the kernels read.
// dst[r * ld + c] = src[r * cols + c]; a non-finite value sets DEVERR_NON_FINITE.
void launch_pack_bf16(const void *src, long long rows, int cols, void *dst, long long ld, cudaStream_t st, DevErr *err);
// The same to float, optionally transposed: dst[c * ld + r].
void launch_expand_f32(const void *src, long long rows, int cols, float *dst, long long ld, bool transpose,
                       cudaStream_t st, DevErr *err);
// dst[offset + r' * row_stride + c' * col_stride] = src[r * cols + c] (bfloat16, or float for Precision::F32) with
// r' = r / row_group * row_pad + r % row_group, and c' alike (group 0: r' = r): rows or columns in padded groups,
// transposed, interleaved.
struct WeightPlace {
  long long offset = 0, row_stride = 0, col_stride = 1;
  int row_group = 0, row_pad = 0, col_group = 0, col_pad = 0;
};
void launch_place(const void *src, long long rows, int cols, void *dst, Precision type, const WeightPlace &at,
                  cudaStream_t st, DevErr *err);
// x <- act(x), or act(x) * factor, on dense float arrays.
void launch_activation_f32(float *x, const float *factor, long long count, Activation act, cudaStream_t st);

}  // namespace lb
