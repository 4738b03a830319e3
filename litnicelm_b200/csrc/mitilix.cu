// The Mitilix decoder: parallel layers (one scalar-gain RMS norm, both sublayers add to the residual
// stream at once), a short causal convolution on each sublayer's input, sliding-window latent attention
// without positions whose latents a layer may take from an earlier one, a dense GELU feed-forward, and
// learned position vectors at the embedding.
//
//   x <- x + ( attention(h + conv1(h)) + down gelu(up (h + conv2(h))) ),   h = rms(x) * gain
//
// State per slot: the latents of every layer that has a down-projection of its own, [slots][cap][rank]
// (a position's row stays where it is, so a layer with a longer window may read a cache that a layer
// with a shorter one fills), and the last taps - 1 rows h of every layer.
//
// A step's launches per layer, bfloat16:
//   few rows    norm + convolutions | W_q, W_dkv and W_up (GELU) in one launch | query and latent store,
//               chunks, join | W_o and W_down as one product over [attention | hidden], added to x
//   many rows   the same with the tensor-core products, and keys and values expanded from the window's
//               latents for the tensor-core attention (V directly transposed, as W_uv c^T)
// 32-bit runs the framework's float products and the CUDA-core attention.
#include "model.cuh"
#include "model_common.cuh"

#include <cmath>
#include <cstring>

namespace lb {

namespace {

struct Layer {
  int heads = 0, dim = 0, vdim = 0, rank = 0, window = 0, kv_from = -1, ff = 0;
  float scale = 0.f, gain = 0.f;
  DevBuf conv1, conv2;     // [taps][width] float
  DevBuf latent_gain;      // [rank] float
  DevBuf uk, uv;           // [heads * dim | vdim, rank]
  DevBuf in, up, out;      // bfloat16: [W_q | pad | W_dkv] [.., width], W_up, [W_o | pad | W_down]
  DevBuf q_t, dkv_t, up_t, o_t, down_t;  // float: transposed to [in, out]
  DevBuf cache, history;
  int q_cols() const { return heads * dim; }
  int o_cols() const { return heads * vdim; }
  bool own() const { return kv_from < 0; }
};

class Mitilix final : public DecoderModel {
 public:
  Mitilix(const Json &c, Precision precision) : prec_(precision) {
    auto size = [](const Json &j, const char *key) {
      const long long v = j.at(key).as_int();
      if (v < 1 || v > (1ll << 30)) throw std::runtime_error(std::string("config: ") + key + " is out of range");
      return (int)v;
    };
    width_ = size(c, "width");
    vocab_ = size(c, "vocab");
    max_positions_ = size(c, "max_positions");
    taps_ = size(c.at("canon"), "taps");
    eps_ = (float)c.at("norm").at("eps").as_number();
    for (const Json &e : c.at("layers").as_array()) {
      const std::string &type = e.at("type").as_string();
      if (type != "latent_attention") throw std::runtime_error("config: unknown mixer \"" + type + "\"");
      const Json &m = e.at("mixer");
      Layer l;
      l.heads = size(m, "heads");
      l.dim = size(m, "dim");
      l.vdim = size(m, "vdim");
      l.rank = size(m, "kv_rank");
      l.scale = (float)m.at("scale").as_number();
      l.window = size(m.at("mask"), "size");
      if (l.window > max_positions_) l.window = max_positions_;
      const int index = (int)layers_.size();
      if (m.has("kv_from")) {
        const long long from = m.at("kv_from").as_int();
        if (from < 0 || from >= index || !layers_[(size_t)from].own() || layers_[(size_t)from].rank != l.rank)
          throw std::runtime_error("config: kv_from of layer " + std::to_string(index) +
                                   " must name an earlier layer with latents of its own and the same kv_rank");
        l.kv_from = (int)from;
      }
      if (e.has("mlp")) {
        const std::string &kind = e.at("mlp").at("kind").as_string();
        if (kind != "dense") throw std::runtime_error("config: unknown feed-forward \"" + kind + "\"");
        l.ff = size(e.at("mlp"), "ff");
      }
      layers_.push_back(std::move(l));
    }
    if (layers_.empty()) throw std::runtime_error("config: no layers");
    for (const Layer &l : layers_) {
      window_max_ = l.window > window_max_ ? l.window : window_max_;
      q_max_ = l.q_cols() > q_max_ ? l.q_cols() : q_max_;
      rank_max_ = l.rank > rank_max_ ? l.rank : rank_max_;
      ff_max_ = l.ff > ff_max_ ? l.ff : ff_max_;
      o_max_ = l.o_cols() > o_max_ ? l.o_cols() : o_max_;
      const int mix = up8(l.o_cols()) + up8(l.ff);
      mix_max_ = mix > mix_max_ ? mix : mix_max_;
    }
  }

  const char *architecture() const override { return "Mitilix"; }
  int n_layers() const override { return (int)layers_.size(); }
  int width() const override { return width_; }
  int vocab() const override { return vocab_; }
  int max_positions() const override { return max_positions_; }
  long long portion_rows() const override { return 32768; }

  int context_bound(int s) const override {
    if (s >= window_max_) return max_positions_;  // every launch has its final size
    int cap = 64;
    while (cap < s) cap *= 2;
    return cap < max_positions_ ? cap : max_positions_;
  }

  void load(const TensorFile &file, cudaStream_t st, DevErr *err) override {
    const int D = width_, V = vocab_, D8 = up8(D);
    DevBuf image;
    image.ensure(file.data_bytes(), st);
    file_to_device(file.path().c_str(), file.data_offset(), file.data_bytes(), image.p, st, false);
    auto at = [&](const std::string &name, std::vector<long long> shape) {
      return static_cast<const void *>(static_cast<const char *>(image.p) + file.bf16(name, shape).begin);
    };
    const bool half = prec_ == Precision::BF16;
    // [rows, cols] into dst (bfloat16, rows ld apart) from element `offset` on
    auto pack = [&](const std::string &name, long long rows, int cols, DevBuf &dst, long long ld, long long offset = 0) {
      launch_pack_bf16(at(name, {rows, cols}), rows, cols, static_cast<uint16_t *>(dst.p) + offset, ld, st, err);
    };
    auto expand = [&](const std::string &name, long long rows, int cols, DevBuf &dst, bool transpose) {
      dst.ensure((size_t)rows * cols * 4, st);
      launch_expand_f32(at(name, {rows, cols}), rows, cols, dst.f(), transpose ? rows : cols, transpose, st, err);
    };
    if (half) {
      embed_.ensure((size_t)V * D * 2, st);
      pos_.ensure((size_t)max_positions_ * D * 2, st);
      head_.ensure((size_t)V * D8 * 2, st);
      pack("embed", V, D, embed_, D);
      pack("pos", max_positions_, D, pos_, D);
      pack("head", V, D, head_, D8);
    } else {
      expand("embed", V, D, embed_, false);
      expand("pos", max_positions_, D, pos_, false);
      expand("head", V, D, head_, true);
    }
    final_gain_ = file.scalar_bf16("final.norm");
    for (size_t i = 0; i < layers_.size(); ++i) {
      Layer &l = layers_[i];
      const std::string p = "l" + std::to_string(i) + ".";
      const int Q = l.q_cols(), O = l.o_cols(), R = l.rank, R8 = up8(R), O8 = up8(O);
      l.gain = file.scalar_bf16(p + "norm1");
      expand(p + "canon1", D, taps_, l.conv1, true);
      if (l.ff) expand(p + "canon2", D, taps_, l.conv2, true);
      if (l.own()) {
        l.latent_gain.ensure((size_t)R * 4, st);
        launch_expand_f32(at(p + "mix.dkv.norm", {R}), 1, R, l.latent_gain.f(), R, false, st, err);
      }
      if (half) {
        l.in.ensure((size_t)(up16(Q) + (l.own() ? R : 0)) * D8 * 2, st);
        pack(p + "mix.q", Q, D, l.in, D8);
        if (l.own()) pack(p + "mix.dkv", R, D, l.in, D8, (long long)up16(Q) * D8);
        l.uk.ensure((size_t)Q * R8 * 2, st);
        l.uv.ensure((size_t)O * R8 * 2, st);
        pack(p + "mix.uk", Q, R, l.uk, R8);
        pack(p + "mix.uv", O, R, l.uv, R8);
        const long long ld = O8 + up8(l.ff);
        l.out.ensure((size_t)D * ld * 2, st);
        pack(p + "mix.o", D, O, l.out, ld);
        if (l.ff) {
          l.up.ensure((size_t)l.ff * D8 * 2, st);
          pack(p + "mlp.up", l.ff, D, l.up, D8);
          pack(p + "mlp.down", D, l.ff, l.out, ld, O8);
        }
      } else {
        expand(p + "mix.q", Q, D, l.q_t, true);
        if (l.own()) expand(p + "mix.dkv", R, D, l.dkv_t, true);
        expand(p + "mix.uk", Q, R, l.uk, false);
        expand(p + "mix.uv", O, R, l.uv, false);
        expand(p + "mix.o", D, O, l.o_t, true);
        if (l.ff) {
          expand(p + "mlp.up", l.ff, D, l.up_t, true);
          expand(p + "mlp.down", D, l.ff, l.down_t, true);
        }
      }
    }
    LB_CUDA(cudaStreamSynchronize(st));
  }

  bool reserve(int streams, int cap, long long rows, cudaStream_t st) override {
    bool moved = false;
    const size_t es = prec_ == Precision::BF16 ? 2 : 4;
    if (streams > slots_ || cap > cap_) {
      const int ns = streams > slots_ ? streams : slots_, nc = cap > cap_ ? cap : cap_;
      for (Layer &l : layers_) {
        const size_t hist = (size_t)(taps_ - 1) * width_ * 4;
        if (ns > slots_ && hist > 0) l.history.grow(hist, slots_, hist, ns, hist, st);
        if (!l.own()) continue;
        const size_t row = (size_t)cache_ld(l) * es;
        l.cache.grow(row * cap_, slots_, row * cap_, ns, row * nc, st);
      }
      slots_ = ns;
      cap_ = nc;
      moved = true;
    }
    if (rows < 8) rows = 8;
    if (rows < streams) rows = streams;
    const size_t R = (size_t)rows;
    moved |= x_.ensure(R * width_ * 4, st);
    moved |= xl_.ensure(R * up8(width_) * es, st);
    moved |= a1_.ensure(R * up8(width_) * es, st);
    moved |= dkv_.ensure(R * rank_max_ * 4, st);
    if (ff_max_ > 0) moved |= a2_.ensure(R * up8(width_) * es, st);
    moved |= q_.ensure(R * up16(q_max_) * es, st);
    if (prec_ == Precision::BF16) {
      moved |= mix_.ensure(R * mix_max_ * 2, st);
      decode_rows_ = slots_ > FEW_ROWS_MAX ? slots_ : FEW_ROWS_MAX;
      size_t need = 0;
      for (const Layer &l : layers_) {
        const size_t n = latent_decode_scratch_floats(l.heads, l.rank, l.window, context_bound(cap_), decode_rows_);
        need = n > need ? n : need;
      }
      moved |= scratch_.ensure(need * 4, st);
    } else {
      moved |= mix_.ensure(R * o_max_ * 4, st);
      if (ff_max_ > 0) moved |= hidden_.ensure(R * ff_max_ * 4, st);
      size_t need = gemv_scratch_floats(8, vocab_, width_);
      for (const Layer &l : layers_)
        for (size_t n : {gemv_scratch_floats(8, l.q_cols(), width_), gemv_scratch_floats(8, l.rank, width_),
                         gemv_scratch_floats(8, width_, l.o_cols()), l.ff ? gemv_scratch_floats(8, l.ff, width_) : 0,
                         l.ff ? gemv_scratch_floats(8, width_, l.ff) : 0})
          need = n > need ? n : need;
      moved |= scratch_.ensure(need * 4 + 16, st);
    }
    return moved;
  }

  int enqueue_rows(const RowBatch &b, cudaStream_t st, DevErr *err) override {
    launches_ = 0;
    launch_embed_rows(embed_.p, pos_.p, 1.0f, prec_, b, width_, vocab_, x_.f(), st, err);
    ++launches_;
    packed_from_ = packed_first_ = -1;
    for (size_t i = 0; i < layers_.size(); ++i) {
      if (prec_ == Precision::BF16) layer_bf16((int)i, b, st, err);
      else layer_f32((int)i, b, st, err);
    }
    return launches_;
  }

  int enqueue_head(const RowBatch &b, const int *rows_dev, int n_rows, float *logits, cudaStream_t st,
                   DevErr *err) override {
    launches_ = 0;
    const int ld = prec_ == Precision::BF16 ? up8(width_) : width_;
    launch_rms_rows(x_.f(), width_, RmsWeight{nullptr, final_gain_}, eps_, rows_dev, n_rows, b.n, xl_.p, ld, prec_, st);
    ++launches_;
    if (prec_ == Precision::BF16) {
      Bf16Product p;
      p.a = xl_.p;
      p.a_ld = ld;
      p.w = head_.p;
      p.w_ld = ld;
      p.n = vocab_;
      p.k = width_;
      p.float_out = logits;
      p.float_ld = vocab_;
      product_bf16(&p, 1, n_rows, st, err);
    } else {
      product_f32(static_cast<float *>(xl_.p), n_rows, width_, head_.f(), vocab_, nullptr, logits, st, err);
    }
    return launches_;
  }

 private:
  int cache_ld(const Layer &l) const { return prec_ == Precision::BF16 ? up8(l.rank) : (l.rank + 3) & ~3; }

  const Layer &source(int i) const {
    const Layer &l = layers_[(size_t)i];
    return l.own() ? l : layers_[(size_t)l.kv_from];
  }

  LatentAttention attention(int i, int w_ld, void *out, int out_ld) const {
    const Layer &l = layers_[(size_t)i];
    LatentAttention a{};
    a.heads = l.heads;
    a.dim = l.dim;
    a.vdim = l.vdim;
    a.scale = l.scale;
    a.window = l.window;
    a.q = q_.p;
    a.q_ld = prec_ == Precision::BF16 ? up16(l.q_cols()) : l.q_cols();
    a.w_uk = l.uk.p;
    a.w_uv = l.uv.p;
    a.w_ld = w_ld;
    a.cache.rows = source(i).cache.p;
    a.cache.cap = cap_;
    a.cache.ld = cache_ld(l);
    a.cache.rank = l.rank;
    a.out = out;
    a.out_ld = out_ld;
    return a;
  }

  void product_bf16(const Bf16Product *p, int count, int m, cudaStream_t st, DevErr *err) {
    launches_ += products_bf16(p, count, m, st, err);
  }

  void layer_bf16(int i, const RowBatch &b, cudaStream_t st, DevErr *err) {
    Layer &l = layers_[(size_t)i];
    const int D = width_, D8 = up8(D), R8 = up8(l.rank), O8 = up8(l.o_cols()), m = (int)b.rows();
    const int mix_ld = O8 + up8(l.ff), q_ld = up16(l.q_cols());
    const CanonConv conv[2] = {{l.conv1.f(), a1_.p, D8}, {l.conv2.f(), a2_.p, D8}};
    launch_rms_canon(x_.f(), D, l.gain, eps_, taps_, l.history.f(), conv, l.ff ? 2 : 1, prec_, b, st);
    ++launches_;
    Bf16Product in[2];
    in[0].a = a1_.p;
    in[0].a_ld = in[0].w_ld = D8;
    in[0].w = l.in.p;
    in[0].k = D;
    in[0].n = l.own() ? q_ld + l.rank : q_ld;
    in[0].n_half = q_ld;
    in[0].half_out = q_.p;
    in[0].half_ld = q_ld;
    in[0].float_out = dkv_.f();
    in[0].float_ld = l.rank;
    in[1].a = a2_.p;
    in[1].a_ld = in[1].w_ld = D8;
    in[1].w = l.up.p;
    in[1].k = D;
    in[1].n = in[1].n_half = l.ff;
    in[1].act = ACT_GELU_ERF;
    in[1].half_out = static_cast<uint16_t *>(mix_.p) + O8;
    in[1].half_ld = mix_ld;
    product_bf16(in, l.ff ? 2 : 1, m, st, err);

    const LatentAttention at = attention(i, R8, mix_.p, mix_ld);
    const bool expand = !(b.n <= 8 || m <= 16) && latent_prefill_supports(l.dim, l.vdim);
    if (expand) {
      // the window's latents side by side (shared with the layers before when they left the same ones)
      const int first = b.p0 - l.window + 1 > 0 ? b.p0 - l.window + 1 : 0;
      const int key_rows = up8(b.p0 + b.n - first), from = l.own() ? i : l.kv_from;
      const long long keys = (long long)b.streams * key_rows;
      if (packed_.ensure((size_t)keys * up8(rank_max_) * 2, st)) packed_from_ = -1;
      k_.ensure((size_t)keys * up8(q_max_) * 2, st);
      vt_.ensure((size_t)o_max_ * up8((int)keys) * 2, st);
      if (l.own() || packed_from_ != from || packed_first_ != first) {
        launch_latent_store(l.own() ? dkv_.f() : nullptr, l.rank, l.latent_gain.f(), eps_, at.cache, packed_.p, key_rows,
                            first, prec_, b, st);
        ++launches_;
        packed_from_ = from;
        packed_first_ = first;
      }
      Bf16Product k;
      k.a = packed_.p;
      k.a_ld = R8;
      k.w = l.uk.p;
      k.w_ld = R8;
      k.n = k.n_half = l.q_cols();
      k.k = l.rank;
      k.half_out = k_.p;
      k.half_ld = up8(l.q_cols());
      launch_gemm_bf16(k, (int)keys, st, err);
      Bf16Product v;  // V^T = W_uv c^T
      v.a = l.uv.p;
      v.a_ld = R8;
      v.w = packed_.p;
      v.w_ld = R8;
      v.n = v.n_half = (int)keys;
      v.k = l.rank;
      v.half_out = vt_.p;
      v.half_ld = up8((int)keys);
      launch_gemm_bf16(v, l.o_cols(), st, err);
      launch_latent_prefill(at, k_.p, up8(l.q_cols()), vt_.p, up8((int)keys), key_rows, first, b, st, err);
      launches_ += 3;
    } else {
      if (m <= decode_rows_ && latent_decode_supports(at)) {
        const LatentFresh fresh{l.own() ? dkv_.f() : nullptr, l.rank, l.latent_gain.f(), eps_};
        launches_ += launch_latent_decode(at, fresh, scratch_.f(), b, st);
      } else {
        if (l.own()) {
          launch_latent_store(dkv_.f(), l.rank, l.latent_gain.f(), eps_, at.cache, nullptr, 0, 0, prec_, b, st);
          ++launches_;
        }
        launch_latent_attention_rows(at, prec_, b, st);
        ++launches_;
      }
    }
    Bf16Product out;
    out.a = mix_.p;
    out.a_ld = out.w_ld = out.k = mix_ld;
    out.w = l.out.p;
    out.n = D;
    out.float_out = x_.f();
    out.float_ld = D;
    out.accumulate = 1;
    product_bf16(&out, 1, m, st, err);
  }

  void product_f32(const float *a, int m, int k, const float *w, int n, const float *residual, float *out,
                   cudaStream_t st, DevErr *err) {
    launches_ += lb::product_f32(a, m, k, w, n, residual, out, scratch_.f(), st, err);
  }

  void layer_f32(int i, const RowBatch &b, cudaStream_t st, DevErr *err) {
    Layer &l = layers_[(size_t)i];
    const int D = width_, m = (int)b.rows();
    const CanonConv conv[2] = {{l.conv1.f(), a1_.p, D}, {l.conv2.f(), a2_.p, D}};
    launch_rms_canon(x_.f(), D, l.gain, eps_, taps_, l.history.f(), conv, l.ff ? 2 : 1, prec_, b, st);
    ++launches_;
    product_f32(a1_.f(), m, D, l.q_t.f(), l.q_cols(), nullptr, q_.f(), st, err);
    const LatentAttention at = attention(i, l.rank, mix_.p, l.o_cols());
    if (l.own()) {
      product_f32(a1_.f(), m, D, l.dkv_t.f(), l.rank, nullptr, dkv_.f(), st, err);
      launch_latent_store(dkv_.f(), l.rank, l.latent_gain.f(), eps_, at.cache, nullptr, 0, 0, prec_, b, st);
      ++launches_;
    }
    launch_latent_attention_rows(at, prec_, b, st);
    ++launches_;
    product_f32(mix_.f(), m, l.o_cols(), l.o_t.f(), D, x_.f(), x_.f(), st, err);
    if (l.ff) {
      product_f32(a2_.f(), m, D, l.up_t.f(), l.ff, nullptr, hidden_.f(), st, err);
      launch_activation_f32(hidden_.f(), nullptr, (long long)m * l.ff, ACT_GELU_ERF, st);
      ++launches_;
      product_f32(hidden_.f(), m, l.ff, l.down_t.f(), D, x_.f(), x_.f(), st, err);
    }
  }

  Precision prec_;
  int width_ = 0, vocab_ = 0, max_positions_ = 0, taps_ = 0;
  float eps_ = 0.f, final_gain_ = 0.f;
  std::vector<Layer> layers_;
  int window_max_ = 1, q_max_ = 0, rank_max_ = 0, ff_max_ = 0, o_max_ = 0, mix_max_ = 0;
  DevBuf embed_, pos_, head_;
  int slots_ = 0, cap_ = 0, launches_ = 0;
  long long decode_rows_ = 0;
  DevBuf x_, xl_, a1_, a2_, q_, dkv_, mix_, hidden_, scratch_;
  DevBuf packed_, k_, vt_;                    // latents, keys and transposed values of a portion's window
  int packed_from_ = -1, packed_first_ = -1;  // whose latents packed_ holds, and from which position on
};

}  // namespace

std::unique_ptr<DecoderModel> make_mitilix(const Json &config, Precision precision) {
  return std::unique_ptr<DecoderModel>(new Mitilix(config, precision));
}

}  // namespace lb
