// The Gobesun decoder: layers of two kinds in any order, each sublayer between two norms,
//
//   x <- x + norm_b(mixer(norm(x)))            mixer: gated delta rule or grouped attention in chunks
//   x <- x + norm_b(down(gelu(gate h) * up h)) h = norm2(x); not every layer has this part
//
// with a run of layers that is gone through several times on the same weights. Every pass of a layer has
// state of its own: per slot the delta rule's [heads][dim][vdim] floats and the convolution's last inputs,
// or the attention's keys and values by position. Nothing is bound to a largest position.
//
// Heads are padded to multiples of 16 elements with zeros, in weights, activations and state: padded
// coordinates stay zero through every step, and the norms count the true ones.
//
// A step's launches per layer, bfloat16:
//   delta      q, k, v, gate, beta and decay in one product | few rows: convolution, recurrence, norm and gate in
//              one kernel; many rows: convolution, chunk matrices, scan | output product
//   attention  q, k, v in one product | norm, rotation, cache | attention | output product
//   mlp        gate and up interleaved in one product whose store applies gelu(gate) * up | down product
// and between any two of them one kernel for both norms and the residual sum. 32-bit runs the framework's
// float products and the same kernels on floats.
#include "model.cuh"
#include "model_common.cuh"

#include <cmath>
#include <cstring>

namespace lb {

namespace {

struct Layer {
  bool delta = false;
  int heads = 0, groups = 0, dim = 0, vdim = 0, ff = 0;
  int dk = 0, dv = 0;  // padded
  // delta
  int taps = 0;
  // attention
  int chunk = 0, rot_dims = 0;
  float scale = 0.f, amplitude = 1.f;
  std::vector<double> turns;  // angle per position over pi
  DevBuf norm1, norm1b, norm2, norm2b;
  DevBuf in, out;             // bfloat16 [n, D8] and [D, heads * dv], float transposed
  DevBuf conv, a_log, dt_bias, head_norm;
  DevBuf q_norm, k_norm, turns_dev;
  DevBuf gate_up, up, down;   // bfloat16: gate and up interleaved in gate_up
  int conv_channels() const { return 2 * groups * dk + heads * dv; }
  int half_cols() const { return delta ? conv_channels() + heads * dv : (heads + groups) * dk + groups * dv; }
  int in_cols() const { return delta ? half_cols() + 2 * heads : half_cols(); }
  int o_cols() const { return heads * dv; }
};

// One pass of a layer: its index and the state of its own.
struct Run {
  int layer = 0;
  DevBuf k_cache, v_cache;  // attention: [slots][cap][groups * dk | dv]
  DevBuf state, history;    // delta: [slots][heads][dk][dv] float, [slots][taps][conv_channels]
};

// Angles per position of every pair: base^(-2 i / dims), the slow pairs divided by `factor` with a ramp between
// the pairs that turn `fast` and `slow` times over `original` positions.
void rotary_turns(const Json &rot, Layer &l) {
  const double base = rot.at("base").as_number();
  const int half = l.rot_dims / 2;
  l.turns.resize((size_t)half);
  for (int i = 0; i < half; ++i) l.turns[(size_t)i] = std::pow(base, -2.0 * i / l.rot_dims);
  if (rot.has("scaling")) {
    const Json &sc = rot.at("scaling");
    const double factor = sc.at("factor").as_number(), original = sc.at("original").as_number();
    auto place = [&](double t) {
      return l.rot_dims * std::log(original / (2.0 * M_PI * t)) / (2.0 * std::log(base));
    };
    const double lo = std::fmax(std::floor(place(sc.at("fast").as_number())), 0.0);
    const double hi = std::fmin(std::ceil(place(sc.at("slow").as_number())), l.rot_dims - 1.0);
    for (int i = 0; i < half; ++i) {
      const double ramp = std::fmin(std::fmax((i - lo) / std::fmax(hi - lo, 0.001), 0.0), 1.0);
      l.turns[(size_t)i] = l.turns[(size_t)i] / factor * ramp + l.turns[(size_t)i] * (1.0 - ramp);
    }
    l.amplitude = (float)(0.1 * std::log(factor) + 1.0);
  }
  for (double &t : l.turns) {
    t /= M_PI;
    if (!std::isfinite(t)) throw std::runtime_error("config: rotary angles are not finite");
  }
}

class Gobesun final : public DecoderModel {
 public:
  Gobesun(const Json &c, Precision precision) : prec_(precision) {
    auto size = [](const Json &j, const char *key) {
      const long long v = j.at(key).as_int();
      if (v < 1 || v > (1ll << 30)) throw std::runtime_error(std::string("config: ") + key + " is out of range");
      return (int)v;
    };
    width_ = size(c, "width");
    vocab_ = size(c, "vocab");
    embed_scale_ = (float)c.at("embedding").at("scale").as_number();
    eps_ = (float)c.at("norm").at("eps").as_number();
    for (const Json &e : c.at("layers").as_array()) {
      const std::string &type = e.at("type").as_string();
      const std::string where = "config: layer " + std::to_string(layers_.size()) + ": ";
      if (type != "delta" && type != "attention") throw std::runtime_error("config: unknown mixer \"" + type + "\"");
      const Json &m = e.at("mixer");
      Layer l;
      l.delta = type == "delta";
      l.heads = size(m, "heads");
      l.groups = size(m, "kv_heads");
      l.dim = size(m, "dim");
      l.vdim = size(m, "vdim");
      if (l.heads % l.groups != 0) throw std::runtime_error(where + "heads is not a multiple of kv_heads");
      l.dk = up16(l.dim);
      l.dv = up16(l.vdim);
      if (l.delta) {
        l.taps = size(m, "conv");
        if (!delta_supports(l.dk, l.dv)) throw std::runtime_error(where + "delta rule heads of this size are not supported");
      } else {
        l.scale = (float)m.at("scale").as_number();
        l.chunk = size(m.at("mask"), "size");
        if (l.dv > 1024) throw std::runtime_error(where + "attention heads of this size are not supported");
        if (m.has("rot")) {
          const long long dims = m.at("rot").at("dims").as_int();
          if (dims < 0 || dims % 2 != 0 || dims > l.dim) throw std::runtime_error(where + "rot.dims must be even and fit the head");
          l.rot_dims = (int)dims;
          rotary_turns(m.at("rot"), l);
        }
        chunk_max_ = l.chunk > chunk_max_ ? l.chunk : chunk_max_;
      }
      if (e.has("mlp")) {
        const std::string &kind = e.at("mlp").at("kind").as_string();
        if (kind != "dense") throw std::runtime_error("config: unknown feed-forward \"" + kind + "\"");
        l.ff = size(e.at("mlp"), "ff");
      }
      layers_.push_back(std::move(l));
    }
    const int n = (int)layers_.size();
    if (n == 0) throw std::runtime_error("config: no layers");
    long long start = 0, stop = 0, times = 1;
    if (c.has("loop")) {
      const Json &loop = c.at("loop");
      start = loop.at("start").as_int();
      stop = loop.at("stop").as_int();
      times = loop.at("times").as_int();
      if (start < 0 || stop < start || stop > n || times < 1 || times * (stop - start) > 100000)
        throw std::runtime_error("config: the loop does not fit the layers");
    }
    std::vector<int> order;
    for (int i = 0; i < start; ++i) order.push_back(i);
    for (int k = 0; k < times; ++k)
      for (int i = (int)start; i < stop; ++i) order.push_back(i);
    for (int i = (int)stop; i < n; ++i) order.push_back(i);
    runs_.resize(order.size());
    for (size_t i = 0; i < order.size(); ++i) runs_[i].layer = order[i];
    for (const Layer &l : layers_) {
      in_max_ = l.in_cols() > in_max_ ? l.in_cols() : in_max_;
      o_max_ = l.o_cols() > o_max_ ? l.o_cols() : o_max_;
      ff_max_ = l.ff > ff_max_ ? l.ff : ff_max_;
      if (!l.delta) q_max_ = l.heads * l.dk > q_max_ ? l.heads * l.dk : q_max_;
      if (l.delta) heads_max_ = l.heads > heads_max_ ? l.heads : heads_max_;
    }
  }

  const char *architecture() const override { return "Gobesun"; }
  int n_layers() const override { return (int)layers_.size(); }
  int width() const override { return width_; }
  int vocab() const override { return vocab_; }
  int max_positions() const override { return 0; }
  long long portion_rows() const override { return 32768; }

  int context_bound(int s) const override {
    if (s >= chunk_max_) return chunk_max_ > 64 ? chunk_max_ : 64;  // no query sees more: every launch has its final size
    int cap = 64;
    while (cap < s) cap *= 2;
    return cap;
  }

  void load(const TensorFile &file, cudaStream_t st, DevErr *err) override {
    const int D = width_, V = vocab_, D8 = up8(D);
    const bool half = prec_ == Precision::BF16;
    const size_t es = half ? 2 : 4;
    DevBuf image;
    image.ensure(file.data_bytes(), st);
    file_to_device(file.path().c_str(), file.data_offset(), file.data_bytes(), image.p, st, false);
    auto at = [&](const std::string &name, std::vector<long long> shape) {
      return static_cast<const void *>(static_cast<const char *>(image.p) + file.bf16(name, shape).begin);
    };
    auto place = [&](const std::string &name, std::vector<long long> shape, DevBuf &dst, Precision type, const WeightPlace &p) {
      const long long rows = shape.size() > 1 ? shape[0] : 1;
      launch_place(at(name, shape), rows, (int)shape.back(), dst.p, type, p, st, err);
    };
    // A vector in float, its groups padded.
    auto vector = [&](const std::string &name, int count, DevBuf &dst, int group = 0, int pad = 0) {
      dst.ensure((size_t)(group ? count / group * pad : count) * 4, st);
      WeightPlace p;
      p.col_group = group;
      p.col_pad = pad;
      place(name, {count}, dst, Precision::F32, p);
    };
    // Product weights [rows, cols] as rows of dst from row `first` on (bfloat16 [n, ld]; float [cols, n] transposed), rows and
    // columns in padded groups, `step` rows apart.
    auto weight = [&](const std::string &name, int rows, int cols, DevBuf &dst, int n, int ld, int first = 0, int row_group = 0,
                      int row_pad = 0, int col_group = 0, int col_pad = 0, int step = 1) {
      const long long wide = col_group ? (long long)cols / col_group * col_pad : cols;
      dst.ensure(half ? (size_t)n * ld * 2 : (size_t)n * wide * 4, st);
      WeightPlace p;
      p.offset = half ? (long long)first * ld : first;
      p.row_stride = (half ? ld : 1) * (long long)step;
      p.col_stride = half ? 1 : n;
      p.row_group = row_group;
      p.row_pad = row_pad;
      p.col_group = col_group;
      p.col_pad = col_pad;
      place(name, {rows, cols}, dst, prec_, p);
    };
    embed_.ensure((size_t)V * D * es, st);
    WeightPlace dense;
    dense.row_stride = D;
    place("embed", {V, D}, embed_, prec_, dense);
    weight("head", V, D, head_, V, D8);
    vector("final.norm", D, final_norm_);
    for (size_t i = 0; i < layers_.size(); ++i) {
      Layer &l = layers_[i];
      const std::string p = "l" + std::to_string(i) + ".", m = p + "mix.";
      const int H = l.heads, G = l.groups, n = in_ld(l);
      vector(p + "norm1", D, l.norm1);
      vector(p + "norm1b", D, l.norm1b);
      const int qh = l.delta ? G : H, vh = l.delta ? H : G, C = l.conv_channels();
      const int k0 = qh * l.dk, v0 = k0 + G * l.dk, g0 = v0 + vh * l.dv;
      const int rows_in = half ? l.in_cols() : n;
      weight(m + "q", qh * l.dim, D, l.in, rows_in, D8, 0, l.dim, l.dk);
      weight(m + "k", G * l.dim, D, l.in, rows_in, D8, k0, l.dim, l.dk);
      weight(m + "v", vh * l.vdim, D, l.in, rows_in, D8, v0, l.vdim, l.dv);
      weight(m + "o", D, H * l.vdim, l.out, D, l.o_cols(), 0, 0, 0, l.vdim, l.dv);
      if (l.delta) {
        weight(m + "g", H * l.vdim, D, l.in, rows_in, D8, g0, l.vdim, l.dv);
        weight(m + "b", H, D, l.in, rows_in, D8, l.half_cols());
        weight(m + "a", H, D, l.in, rows_in, D8, l.half_cols() + H);
        l.conv.ensure((size_t)l.taps * C * 4, st);
        auto conv = [&](const std::string &name, int channels, int group, int pad, int first) {
          WeightPlace w;
          w.offset = first;
          w.row_stride = 1;
          w.col_stride = C;
          w.row_group = group;
          w.row_pad = pad;
          place(name, {channels, l.taps}, l.conv, Precision::F32, w);
        };
        conv(m + "q.conv", G * l.dim, l.dim, l.dk, 0);
        conv(m + "k.conv", G * l.dim, l.dim, l.dk, k0);
        conv(m + "v.conv", H * l.vdim, l.vdim, l.dv, v0);
        vector(m + "A_log", H, l.a_log);
        vector(m + "dt_bias", H, l.dt_bias);
        vector(m + "norm", l.vdim, l.head_norm, l.vdim, l.dv);
      } else {
        vector(m + "q.norm", H * l.dim, l.q_norm, l.dim, l.dk);
        vector(m + "k.norm", G * l.dim, l.k_norm, l.dim, l.dk);
        l.turns_dev.ensure(l.turns.size() * 8 + 8, st);
        if (!l.turns.empty())
          LB_CUDA(cudaMemcpyAsync(l.turns_dev.p, l.turns.data(), l.turns.size() * 8, cudaMemcpyHostToDevice, st));
      }
      if (l.ff) {
        vector(p + "norm2", D, l.norm2);
        vector(p + "norm2b", D, l.norm2b);
        if (half) {
          weight(p + "mlp.gate", l.ff, D, l.gate_up, 2 * l.ff, D8, 0, 0, 0, 0, 0, 2);
          weight(p + "mlp.up", l.ff, D, l.gate_up, 2 * l.ff, D8, 1, 0, 0, 0, 0, 2);
        } else {
          weight(p + "mlp.gate", l.ff, D, l.gate_up, l.ff, D8);
          weight(p + "mlp.up", l.ff, D, l.up, l.ff, D8);
        }
        weight(p + "mlp.down", D, l.ff, l.down, D, up8(l.ff));
      }
    }
    LB_CUDA(cudaStreamSynchronize(st));
  }

  bool reserve(int streams, int cap, long long rows, cudaStream_t st) override {
    bool moved = false;
    const size_t es = prec_ == Precision::BF16 ? 2 : 4;
    if (streams > slots_ || cap > cap_) {
      const int ns = streams > slots_ ? streams : slots_, nc = cap > cap_ ? cap : cap_;
      for (Run &r : runs_) {
        const Layer &l = layers_[(size_t)r.layer];
        if (l.delta) {
          if (ns == slots_) continue;
          const size_t state = (size_t)l.heads * l.dk * l.dv * 4, hist = (size_t)l.taps * l.conv_channels() * es;
          r.state.grow(state, slots_, state, ns, state, st);
          r.history.grow(hist, slots_, hist, ns, hist, st);
        } else {
          const size_t k = (size_t)l.groups * l.dk * es, v = (size_t)l.groups * l.dv * es;
          r.k_cache.grow(k * cap_, slots_, k * cap_, ns, k * nc, st);
          r.v_cache.grow(v * cap_, slots_, v * cap_, ns, v * nc, st);
        }
      }
      slots_ = ns;
      cap_ = nc;
      moved = true;
    }
    if (rows < 8) rows = 8;
    if (rows < streams) rows = streams;
    const size_t R = (size_t)rows;
    moved |= x_.ensure(R * width_ * 4, st);
    moved |= y_.ensure(R * width_ * 4, st);
    moved |= h_.ensure(R * up8(width_) * es, st);
    moved |= in_.ensure(R * up8(in_max_) * es, st);
    moved |= mix_.ensure(R * o_max_ * es, st);
    if (heads_max_ > 0 && prec_ == Precision::BF16) moved |= ba_.ensure(R * 2 * heads_max_ * 4, st);
    if (q_max_ > 0) moved |= q_.ensure(R * q_max_ * es, st);
    if (ff_max_ > 0) moved |= hidden_.ensure(R * up8(ff_max_) * es, st);
    size_t need = 0;
    auto most = [&](size_t n) { need = n > need ? n : need; };
    for (const Layer &l : layers_)
      if (l.delta) {
        DeltaMixer m{};
        sizes(l, m);
        most(delta_scratch_bytes(m, rows, slots_, prec_));
      }
    if (need > 0) moved |= delta_.ensure(need, st);
    if (prec_ == Precision::F32) {
      if (ff_max_ > 0) moved |= factor_.ensure(R * ff_max_ * 4, st);
      need = gemv_scratch_floats(8, vocab_, width_);
      for (const Layer &l : layers_) {
        most(gemv_scratch_floats(8, in_ld(l), width_));
        most(gemv_scratch_floats(8, width_, l.o_cols()));
        if (l.ff) {
          most(gemv_scratch_floats(8, l.ff, width_));
          most(gemv_scratch_floats(8, width_, l.ff));
        }
      }
      moved |= scratch_.ensure(need * 4 + 16, st);
    }
    return moved;
  }

  int enqueue_rows(const RowBatch &b, cudaStream_t st, DevErr *err) override {
    launches_ = 0;
    launch_embed_rows(embed_.p, nullptr, embed_scale_, prec_, b, width_, vocab_, x_.f(), st, err);
    ++launches_;
    norms(nullptr, nullptr, &layers_[(size_t)runs_[0].layer].norm1, b, st);
    for (size_t i = 0; i < runs_.size(); ++i) {
      Run &r = runs_[i];
      const Layer &l = layers_[(size_t)r.layer];
      const DevBuf *next = i + 1 < runs_.size() ? &layers_[(size_t)runs_[i + 1].layer].norm1 : nullptr;
      if (l.delta) delta(l, r, b, st, err);
      else attention(l, r, b, st, err);
      product(mix_.p, l.o_cols(), l.o_cols(), l.out, width_, y_.f(), b, st, err);
      norms(y_.f(), &l.norm1b, l.ff ? &l.norm2 : next, b, st);
      if (l.ff) {
        feed_forward(l, b, st, err);
        norms(y_.f(), &l.norm2b, next, b, st);
      }
    }
    return launches_;
  }

  int enqueue_head(const RowBatch &b, const int *rows_dev, int n_rows, float *logits, cudaStream_t st,
                   DevErr *err) override {
    launches_ = 0;
    launch_rms_rows(x_.f(), width_, RmsWeight{final_norm_.f(), 1.f}, eps_, rows_dev, n_rows, b.n, h_.p, h_ld(), prec_, st);
    ++launches_;
    product(h_.p, h_ld(), width_, head_, vocab_, logits, n_rows, st, err);
    return launches_;
  }

 private:
  int h_ld() const { return prec_ == Precision::BF16 ? up8(width_) : width_; }
  // Columns of a projected row as stored.
  int in_ld(const Layer &l) const { return prec_ == Precision::BF16 ? l.half_cols() : up8(l.in_cols()); }

  // x <- x + rms(y) (1 + after), h = rms(x) (1 + before)
  void norms(const float *y, const DevBuf *after, const DevBuf *before, const RowBatch &b, cudaStream_t st) {
    launch_residual_norm(x_.f(), y, RmsWeight{after ? after->f() : nullptr, 1.f}, before ? h_.p : nullptr, h_ld(),
                         RmsWeight{before ? before->f() : nullptr, 1.f}, width_, b.rows(), eps_, prec_, st);
    ++launches_;
  }

  // out[m, n] = a[m, k] w^T in float
  void product(const void *a, int a_ld, int k, const DevBuf &w, int n, float *out, int m, cudaStream_t st, DevErr *err) {
    if (prec_ == Precision::F32) {
      launches_ += product_f32(static_cast<const float *>(a), m, k, w.f(), n, nullptr, out, scratch_.f(), st, err);
      return;
    }
    Bf16Product p;
    p.a = a;
    p.a_ld = p.w_ld = a_ld;
    p.w = w.p;
    p.n = n;
    p.k = k;
    p.float_out = out;
    p.float_ld = n;
    launches_ += products_bf16(&p, 1, m, st, err);
  }
  void product(const void *a, int a_ld, int k, const DevBuf &w, int n, float *out, const RowBatch &b, cudaStream_t st,
               DevErr *err) {
    product(a, a_ld, k, w, n, out, (int)b.rows(), st, err);
  }

  // The layer's projections of h into in_ (and ba_).
  void project(const Layer &l, const RowBatch &b, cudaStream_t st, DevErr *err) {
    const int m = (int)b.rows();
    if (prec_ == Precision::F32) {
      launches_ += product_f32(h_.f(), m, width_, l.in.f(), in_ld(l), nullptr, in_.f(), scratch_.f(), st, err);
      return;
    }
    Bf16Product p;
    p.a = h_.p;
    p.a_ld = p.w_ld = h_ld();
    p.w = l.in.p;
    p.n = l.in_cols();
    p.k = width_;
    p.n_half = l.half_cols();
    p.half_out = in_.p;
    p.half_ld = in_ld(l);
    p.float_out = ba_.f();
    p.float_ld = 2 * l.heads;
    launches_ += products_bf16(&p, 1, m, st, err);
  }

  void sizes(const Layer &l, DeltaMixer &m) const {
    m.heads = l.heads;
    m.groups = l.groups;
    m.dim = l.dk;
    m.vdim = l.dv;
    m.true_dim = l.dim;
    m.true_vdim = l.vdim;
    m.taps = l.taps;
  }

  void delta(const Layer &l, Run &r, const RowBatch &b, cudaStream_t st, DevErr *err) {
    project(l, b, st, err);
    DeltaMixer m{};
    sizes(l, m);
    m.eps = eps_;
    m.conv = l.conv.f();
    m.a_log = l.a_log.f();
    m.dt_bias = l.dt_bias.f();
    m.norm = l.head_norm.f();
    m.state = r.state.f();
    m.history = r.history.p;
    m.in = in_.p;
    m.in_ld = in_ld(l);
    const bool half = prec_ == Precision::BF16;
    m.ba = half ? ba_.f() : in_.f() + l.half_cols();
    m.ba_ld = half ? 2 * l.heads : m.in_ld;
    m.out = mix_.p;
    m.out_ld = l.o_cols();
    launches_ += launch_delta(m, delta_.p, prec_, b, st, err);
  }

  void attention(const Layer &l, Run &r, const RowBatch &b, cudaStream_t st, DevErr *err) {
    project(l, b, st, err);
    GroupedAttention a{};
    a.heads = l.heads;
    a.groups = l.groups;
    a.dim = l.dk;
    a.vdim = l.dv;
    a.scale = l.scale;
    a.span.kind = SpanKind::CHUNK;
    a.span.size = l.chunk;
    a.q = q_.p;
    a.q_ld = l.heads * l.dk;
    a.k_cache = r.k_cache.p;
    a.v_cache = r.v_cache.p;
    a.cap = cap_;
    a.slots = slots_;
    a.out = mix_.p;
    a.out_ld = l.o_cols();
    Rotation rot;
    rot.dims = l.rot_dims;
    rot.turns = static_cast<const double *>(l.turns_dev.p);
    rot.amplitude = l.amplitude;
    launch_qk_norm_rotate(in_.p, in_ld(l), l.q_norm.f(), l.k_norm.f(), eps_, l.dim, rot, a, q_.p, prec_, b, st);
    const bool many = b.n > 8 && b.rows() > 16;
    if (prec_ == Precision::BF16 && many && grouped_prefill_supports(l.dk, l.dv)) launch_grouped_prefill(a, b, st, err);
    else launch_grouped_attention_rows(a, prec_, b, st);
    launches_ += 2;
  }

  void feed_forward(const Layer &l, const RowBatch &b, cudaStream_t st, DevErr *err) {
    const int m = (int)b.rows();
    if (prec_ == Precision::F32) {
      launches_ += product_f32(h_.f(), m, width_, l.gate_up.f(), l.ff, nullptr, hidden_.f(), scratch_.f(), st, err);
      launches_ += product_f32(h_.f(), m, width_, l.up.f(), l.ff, nullptr, factor_.f(), scratch_.f(), st, err);
      launch_activation_f32(hidden_.f(), factor_.f(), (long long)m * l.ff, ACT_GELU_TANH, st);
      ++launches_;
      product(hidden_.p, l.ff, l.ff, l.down, width_, y_.f(), m, st, err);
      return;
    }
    Bf16Product p;
    p.a = h_.p;
    p.a_ld = p.w_ld = h_ld();
    p.w = l.gate_up.p;
    p.n = p.n_half = 2 * l.ff;
    p.k = width_;
    p.act = ACT_GELU_TANH;
    p.gated = 1;
    p.half_out = hidden_.p;
    p.half_ld = up8(l.ff);
    launches_ += products_bf16(&p, 1, m, st, err);
    product(hidden_.p, up8(l.ff), l.ff, l.down, width_, y_.f(), m, st, err);
  }

  Precision prec_;
  int width_ = 0, vocab_ = 0, chunk_max_ = 1;
  float eps_ = 0.f, embed_scale_ = 1.f;
  std::vector<Layer> layers_;
  std::vector<Run> runs_;
  int in_max_ = 0, o_max_ = 0, ff_max_ = 0, q_max_ = 0, heads_max_ = 0;
  DevBuf embed_, head_, final_norm_;
  int slots_ = 0, cap_ = 0, launches_ = 0;
  DevBuf x_, y_, h_, in_, ba_, q_, mix_, hidden_, factor_, delta_, scratch_;
};

}  // namespace

std::unique_ptr<DecoderModel> make_gobesun(const Json &config, Precision precision) {
  return std::unique_ptr<DecoderModel>(new Gobesun(config, precision));
}

}  // namespace lb
