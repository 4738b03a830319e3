// Single operators of the registered decoder designs on host buffers, for checking each against an
// independent implementation. Every call allocates and frees its own device memory.
#include "model.cuh"
#include "gemm_tc.cuh"

#include <algorithm>
#include <cstring>
#include <vector>

namespace lb {
namespace {

struct Dev {
  std::vector<void *> all;
  ~Dev() {
    for (void *p : all) cudaFree(p);
  }
  void *alloc(size_t bytes) {
    void *p = nullptr;
    if (cudaMalloc(&p, bytes + 256) != cudaSuccess) throw std::bad_alloc();
    all.push_back(p);
    LB_CUDA(cudaMemset(p, 0, bytes + 256));
    return p;
  }
};

uint16_t to_bf16(float v) {
  uint32_t u;
  std::memcpy(&u, &v, 4);
  return (uint16_t)((u + 0x7fffu + ((u >> 16) & 1u)) >> 16);
}
float from_bf16(uint16_t h) {
  const uint32_t u = (uint32_t)h << 16;
  float v;
  std::memcpy(&v, &u, 4);
  return v;
}

// Host [rows, cols] floats -> device rows ld elements apart, bfloat16 or float.
void *put(Dev &dev, const float *src, long long rows, int cols, int ld, Precision type) {
  const size_t es = type == Precision::BF16 ? 2 : 4;
  std::vector<unsigned char> h((size_t)rows * ld * es, 0);
  for (long long r = 0; r < rows; ++r)
    for (int c = 0; c < cols; ++c) {
      const float v = src[r * cols + c];
      if (es == 2) {
        const uint16_t b = to_bf16(v);
        std::memcpy(&h[((size_t)r * ld + c) * 2], &b, 2);
      } else {
        std::memcpy(&h[((size_t)r * ld + c) * 4], &v, 4);
      }
    }
  void *p = dev.alloc(h.size());
  LB_CUDA(cudaMemcpy(p, h.data(), h.size(), cudaMemcpyHostToDevice));
  return p;
}

void get(const void *src, long long rows, int cols, int ld, Precision type, float *dst) {
  const size_t es = type == Precision::BF16 ? 2 : 4;
  std::vector<unsigned char> h((size_t)rows * ld * es);
  LB_CUDA(cudaMemcpy(h.data(), src, h.size(), cudaMemcpyDeviceToHost));
  for (long long r = 0; r < rows; ++r)
    for (int c = 0; c < cols; ++c) {
      if (es == 2) {
        uint16_t b;
        std::memcpy(&b, &h[((size_t)r * ld + c) * 2], 2);
        dst[r * cols + c] = from_bf16(b);
      } else {
        std::memcpy(&dst[r * cols + c], &h[((size_t)r * ld + c) * 4], 4);
      }
    }
}

struct ErrWord {
  DevErr *host = nullptr, *dev = nullptr;
  ErrWord() {
    LB_CUDA(cudaHostAlloc(reinterpret_cast<void **>(&host), sizeof(DevErr), cudaHostAllocMapped));
    host->code = host->detail = 0;
    LB_CUDA(cudaHostGetDevicePointer(reinterpret_cast<void **>(&dev), host, 0));
  }
  ~ErrWord() { cudaFreeHost(host); }
};

template <class Fn>
int diag(Fn fn) {
  try {
    return fn();
  } catch (const std::bad_alloc &) {
    return LITNICE_B200_ENOMEM;
  } catch (const CudaError &) {
    return LITNICE_B200_ECUDA;
  } catch (const std::exception &) {
    return LITNICE_B200_EINVAL;
  }
}

int up8(int v) { return (v + 7) & ~7; }
int up16(int v) { return (v + 15) & ~15; }

}  // namespace
}  // namespace lb

using namespace lb;

extern "C" {

int litnice_b200_bf16_product_host(int32_t engine, const float *a, int32_t m, int32_t k, const float *w, int32_t n,
                                   int32_t n_half, int32_t act, int32_t gated, int32_t accumulate, float *c) {
  return diag([&]() {
    if (a == nullptr || w == nullptr || c == nullptr || m <= 0 || k <= 0 || n <= 0 || n_half < 0 || n_half > n ||
        (engine == 0 && m > FEW_ROWS_MAX) || engine < 0 || engine > 1 || act < ACT_NONE || act > ACT_GELU_TANH ||
        (gated && n_half % 2 != 0))
      return LITNICE_B200_EINVAL;
    Dev dev;
    ErrWord err;
    const int ld = up8(k), nf = n - n_half, nh = gated ? n_half / 2 : n_half;
    Bf16Product p;
    p.a = put(dev, a, m, k, ld, Precision::BF16);
    p.w = put(dev, w, n, k, ld, Precision::BF16);
    p.a_ld = p.w_ld = ld;
    p.n = n;
    p.k = k;
    p.n_half = n_half;
    p.half_out = dev.alloc((size_t)m * up8(nh ? nh : 1) * 2);
    p.half_ld = up8(nh ? nh : 1);
    p.act = act;
    p.gated = gated;
    p.float_ld = nf > 0 ? nf : 1;
    p.accumulate = accumulate;
    std::vector<float> part((size_t)m * (nf > 0 ? nf : 1));
    for (int r = 0; r < m; ++r)
      for (int j = 0; j < nf; ++j) part[(size_t)r * nf + j] = c[(size_t)r * (nh + nf) + nh + j];
    p.float_out = static_cast<float *>(put(dev, part.data(), m, p.float_ld, p.float_ld, Precision::F32));
    if (engine == 0) launch_few_row_bf16(&p, 1, m, nullptr);
    else launch_gemm_bf16(p, m, nullptr, err.dev);
    LB_CUDA(cudaDeviceSynchronize());
    if (err.host->code != DEVERR_NONE) return LITNICE_B200_EDEVICE;
    std::vector<float> half((size_t)m * (nh ? nh : 1));
    if (nh) get(p.half_out, m, nh, p.half_ld, Precision::BF16, half.data());
    get(p.float_out, m, p.float_ld, p.float_ld, Precision::F32, part.data());
    for (int r = 0; r < m; ++r)
      for (int j = 0; j < nh + nf; ++j)
        c[(size_t)r * (nh + nf) + j] = j < nh ? half[(size_t)r * nh + j] : part[(size_t)r * nf + j - nh];
    return LITNICE_B200_OK;
  });
}

int litnice_b200_rms_canon_host(int32_t dtype, const float *x, int32_t n, int32_t d, float gain, float eps, int32_t taps,
                                const float *w1, const float *w2, const int32_t *portions, int32_t n_portions, float *out1,
                                float *out2) {
  return diag([&]() {
    if (x == nullptr || w1 == nullptr || out1 == nullptr || (w2 != nullptr) != (out2 != nullptr) || n <= 0 || d <= 0 ||
        taps < 1 || portions == nullptr || n_portions <= 0)
      return LITNICE_B200_EINVAL;
    int total = 0;
    for (int i = 0; i < n_portions; ++i) {
      if (portions[i] <= 0 || portions[i] > n - total) return LITNICE_B200_EINVAL;
      total += portions[i];
    }
    if (total != n) return LITNICE_B200_EINVAL;
    const Precision type = dtype == LITNICE_B200_DTYPE_F32 ? Precision::F32 : Precision::BF16;
    Dev dev;
    const int ld = up8(d);
    float *hist = static_cast<float *>(dev.alloc((size_t)(taps - 1) * d * 4));
    // what an earlier sequence may have left in the slot
    LB_CUDA(cudaMemset(hist, 0x41, (size_t)(taps - 1) * d * 4));
    auto transposed = [&](const float *w) {
      std::vector<float> t((size_t)taps * d);
      for (int c = 0; c < d; ++c)
        for (int j = 0; j < taps; ++j) t[(size_t)j * d + c] = w[(size_t)c * taps + j];
      return static_cast<float *>(put(dev, t.data(), taps, d, d, Precision::F32));
    };
    CanonConv conv[2];
    conv[0].w = transposed(w1);
    if (w2) conv[1].w = transposed(w2);
    for (int i = 0, p0 = 0; i < n_portions; p0 += portions[i], ++i) {
      RowBatch b;
      b.p0 = p0;
      b.n = portions[i];
      b.s_cap = p0 + b.n;
      const float *xd = static_cast<float *>(put(dev, x + (size_t)p0 * d, b.n, d, d, Precision::F32));
      for (CanonConv &c : conv) {
        c.out = dev.alloc((size_t)b.n * ld * 4);
        c.ld = ld;
      }
      launch_rms_canon(xd, d, gain, eps, taps, hist, conv, w2 ? 2 : 1, type, b, nullptr);
      LB_CUDA(cudaDeviceSynchronize());
      get(conv[0].out, b.n, d, ld, type, out1 + (size_t)p0 * d);
      if (w2) get(conv[1].out, b.n, d, ld, type, out2 + (size_t)p0 * d);
    }
    return LITNICE_B200_OK;
  });
}

int litnice_b200_latent_attention_host(int32_t engine, const float *q, const float *dkv, const float *latent_gain,
                                       float eps, const float *w_uk, const float *w_uv, int32_t n_streams, int32_t p0,
                                       int32_t n, int32_t heads, int32_t dim, int32_t vdim, int32_t rank, float scale,
                                       int32_t window, float *out) {
  return diag([&]() {
    if (q == nullptr || dkv == nullptr || latent_gain == nullptr || w_uk == nullptr || w_uv == nullptr || out == nullptr ||
        n_streams <= 0 || p0 < 0 || n <= 0 || heads <= 0 || dim <= 0 || vdim <= 0 || rank <= 0 || window <= 0)
      return LITNICE_B200_EINVAL;
    if (engine < 0 || engine > 3) return LITNICE_B200_EINVAL;
    const Precision type = engine == 0 ? Precision::F32 : Precision::BF16;
    const size_t es = type == Precision::BF16 ? 2 : 4;
    if (engine == 3 && !latent_prefill_supports(dim, vdim)) return LITNICE_B200_EINVAL;
    Dev dev;
    ErrWord err;
    const int T = p0 + n, ld = up8(rank), hd = heads * dim, hv = heads * vdim;
    const float *gain = static_cast<float *>(put(dev, latent_gain, 1, rank, rank, Precision::F32));
    LatentAttention a{};
    a.heads = heads;
    a.dim = dim;
    a.vdim = vdim;
    a.scale = scale;
    a.window = window;
    a.q = put(dev, q, (long long)n_streams * n, hd, up8(hd), type);
    a.q_ld = up8(hd);
    a.w_uk = put(dev, w_uk, hd, rank, ld, type);
    a.w_uv = put(dev, w_uv, hv, rank, ld, type);
    a.w_ld = ld;
    a.cache.rows = dev.alloc((size_t)n_streams * T * ld * es);
    a.cache.cap = T;
    a.cache.ld = ld;
    a.cache.rank = rank;
    a.out = dev.alloc((size_t)n_streams * n * up8(hv) * es);
    a.out_ld = up8(hv);
    RowBatch past, b;  // dkv [n_streams, T, rank]: the rows before p0 fill the cache first
    past.streams = b.streams = n_streams;
    std::vector<float> rows;
    auto slice = [&](int from, int count) {
      rows.resize((size_t)n_streams * count * rank);
      for (int s = 0; s < n_streams; ++s)
        std::memcpy(&rows[(size_t)s * count * rank], dkv + ((size_t)s * T + from) * rank, (size_t)count * rank * 4);
      return static_cast<float *>(put(dev, rows.data(), (long long)n_streams * count, rank, rank, Precision::F32));
    };
    if (p0 > 0) {
      past.p0 = 0;
      past.n = past.s_cap = p0;
      launch_latent_store(slice(0, p0), rank, gain, eps, a.cache, nullptr, 0, 0, type, past, nullptr);
    }
    b.p0 = p0;
    b.n = n;
    b.s_cap = T;
    const float *fresh = slice(p0, n);
    if (engine <= 2) {
      if (engine != 2) launch_latent_store(fresh, rank, gain, eps, a.cache, nullptr, 0, 0, type, b, nullptr);
      if (engine == 2) {
        if (!latent_decode_supports(a)) return LITNICE_B200_EINVAL;
        float *scratch = static_cast<float *>(
            dev.alloc(latent_decode_scratch_floats(heads, rank, window, T, b.rows()) * 4));
        launch_latent_decode(a, LatentFresh{fresh, rank, gain, eps}, scratch, b, nullptr);
      } else {
        launch_latent_attention_rows(a, type, b, nullptr);
      }
    } else {
      const int first = p0 - window + 1 > 0 ? p0 - window + 1 : 0, key_rows = up8(T - first);
      const long long keys = (long long)n_streams * key_rows;
      void *packed = dev.alloc((size_t)keys * ld * 2), *k = dev.alloc((size_t)keys * up8(hd) * 2),
           *vt = dev.alloc((size_t)hv * up8((int)keys) * 2);
      launch_latent_store(fresh, rank, gain, eps, a.cache, packed, key_rows, first, type, b, nullptr);
      Bf16Product p;
      p.a = packed;
      p.a_ld = p.w_ld = ld;
      p.w = a.w_uk;
      p.n = p.n_half = hd;
      p.k = rank;
      p.half_out = k;
      p.half_ld = up8(hd);
      launch_gemm_bf16(p, (int)keys, nullptr, err.dev);
      p.a = a.w_uv;
      p.w = packed;
      p.n = p.n_half = (int)keys;
      p.half_out = vt;
      p.half_ld = up8((int)keys);
      launch_gemm_bf16(p, hv, nullptr, err.dev);
      launch_latent_prefill(a, k, up8(hd), vt, up8((int)keys), key_rows, first, b, nullptr, err.dev);
    }
    LB_CUDA(cudaDeviceSynchronize());
    if (err.host->code != DEVERR_NONE) return LITNICE_B200_EDEVICE;
    get(a.out, (long long)n_streams * n, hv, up8(hv), type, out);
    return LITNICE_B200_OK;
  });
}

int litnice_b200_residual_norm_host(int32_t dtype, float *x, const float *y, const float *after, const float *before,
                                    float base, int32_t n, int32_t d, float eps, float *h) {
  return diag([&]() {
    if (x == nullptr || n <= 0 || d <= 0 || (y != nullptr && after == nullptr) || (h != nullptr && before == nullptr))
      return LITNICE_B200_EINVAL;
    const Precision type = dtype == LITNICE_B200_DTYPE_F32 ? Precision::F32 : Precision::BF16;
    Dev dev;
    const int ld = up8(d);
    auto floats = [&](const float *p, int rows) {
      return p ? static_cast<float *>(put(dev, p, rows, d, d, Precision::F32)) : nullptr;
    };
    float *xd = floats(x, n);
    void *hd = h ? dev.alloc((size_t)n * ld * 4) : nullptr;
    launch_residual_norm(xd, floats(y, n), RmsWeight{floats(after, 1), base}, hd, ld, RmsWeight{floats(before, 1), base}, d, n,
                         eps, type, nullptr);
    LB_CUDA(cudaDeviceSynchronize());
    get(xd, n, d, d, Precision::F32, x);
    if (h) get(hd, n, d, ld, type, h);
    return LITNICE_B200_OK;
  });
}

int litnice_b200_delta_host(int32_t dtype, const float *rows, const float *ba, const float *conv, const float *a_log,
                            const float *dt_bias, const float *norm, float eps, int32_t n_streams, int32_t n, int32_t heads,
                            int32_t groups, int32_t dim, int32_t vdim, int32_t taps, const int32_t *portions,
                            int32_t n_portions, float *out, float *state) {
  return diag([&]() {
    if (rows == nullptr || ba == nullptr || conv == nullptr || a_log == nullptr || dt_bias == nullptr || norm == nullptr ||
        out == nullptr || state == nullptr || portions == nullptr || n_streams <= 0 || n <= 0 || heads <= 0 || groups <= 0 ||
        heads % groups != 0 || dim <= 0 || vdim <= 0 || taps <= 0 || n_portions <= 0)
      return LITNICE_B200_EINVAL;
    int total = 0;
    for (int i = 0; i < n_portions; ++i) {
      if (portions[i] <= 0 || portions[i] > n - total) return LITNICE_B200_EINVAL;
      total += portions[i];
    }
    if (total != n) return LITNICE_B200_EINVAL;
    const Precision type = dtype == LITNICE_B200_DTYPE_F32 ? Precision::F32 : Precision::BF16;
    const size_t es = type == Precision::BF16 ? 2 : 4;
    Dev dev;
    ErrWord err;
    DeltaMixer m{};
    m.heads = heads;
    m.groups = groups;
    m.true_dim = dim;
    m.true_vdim = vdim;
    m.dim = up16(dim);
    m.vdim = up16(vdim);
    m.taps = taps;
    m.eps = eps;
    if (!delta_supports(m.dim, m.vdim)) return LITNICE_B200_EINVAL;
    const int C = m.conv_channels(), W = C + heads * m.vdim, true_c = 2 * groups * dim + heads * vdim,
              true_w = true_c + heads * vdim;
    // column of a true column, in rows of padded heads
    auto column = [&](int c) {
      if (c < 2 * groups * dim) return c / dim * m.dim + c % dim;
      c -= 2 * groups * dim;
      return 2 * groups * m.dim + c / vdim * m.vdim + c % vdim;
    };
    std::vector<float> wide((size_t)taps * C, 0.f);
    for (int c = 0; c < true_c; ++c)
      for (int j = 0; j < taps; ++j) wide[(size_t)j * C + column(c)] = conv[(size_t)c * taps + j];
    m.conv = static_cast<float *>(put(dev, wide.data(), taps, C, C, Precision::F32));
    m.a_log = static_cast<float *>(put(dev, a_log, 1, heads, heads, Precision::F32));
    m.dt_bias = static_cast<float *>(put(dev, dt_bias, 1, heads, heads, Precision::F32));
    std::vector<float> gain((size_t)m.vdim, 0.f);
    std::copy(norm, norm + vdim, gain.begin());
    m.norm = static_cast<float *>(put(dev, gain.data(), 1, m.vdim, m.vdim, Precision::F32));
    const int slot0 = 1, slots = n_streams + slot0;
    const size_t state_bytes = (size_t)slots * heads * m.dim * m.vdim * 4, hist_bytes = (size_t)slots * taps * C * es;
    m.state = static_cast<float *>(dev.alloc(state_bytes));
    m.history = dev.alloc(hist_bytes);
    LB_CUDA(cudaMemset(m.state, 0x41, state_bytes));  // what an earlier sequence may have left in the slots
    LB_CUDA(cudaMemset(m.history, 0x41, hist_bytes));
    m.in_ld = W;
    m.out_ld = heads * m.vdim;
    m.ba_ld = 2 * heads;
    for (int i = 0, p0 = 0; i < n_portions; p0 += portions[i], ++i) {
      RowBatch b;
      b.streams = n_streams;
      b.slot0 = slot0;
      b.p0 = p0;
      b.n = portions[i];
      b.s_cap = p0 + b.n;
      std::vector<float> in((size_t)b.rows() * W, 0.f), gates((size_t)b.rows() * 2 * heads);
      for (int st = 0; st < n_streams; ++st)
        for (int t = 0; t < b.n; ++t) {
          const size_t r = (size_t)st * b.n + t, src = (size_t)st * n + p0 + t;
          for (int c = 0; c < true_w; ++c) in[r * W + column(c)] = rows[src * true_w + c];
          std::copy(ba + src * 2 * heads, ba + (src + 1) * 2 * heads, gates.begin() + r * 2 * heads);
        }
      m.in = put(dev, in.data(), b.rows(), W, W, type);
      m.ba = static_cast<float *>(put(dev, gates.data(), b.rows(), 2 * heads, 2 * heads, Precision::F32));
      m.out = dev.alloc((size_t)b.rows() * m.out_ld * es);
      void *scratch = dev.alloc(delta_scratch_bytes(m, b.rows(), n_streams, type));
      launch_delta(m, scratch, type, b, nullptr, err.dev);
      LB_CUDA(cudaDeviceSynchronize());
      if (err.host->code != DEVERR_NONE) return LITNICE_B200_EDEVICE;
      std::vector<float> o((size_t)b.rows() * m.out_ld);
      get(m.out, b.rows(), m.out_ld, m.out_ld, type, o.data());
      for (int st = 0; st < n_streams; ++st)
        for (int t = 0; t < b.n; ++t)
          for (int h = 0; h < heads; ++h)
            for (int e = 0; e < vdim; ++e)
              out[(((size_t)st * n + p0 + t) * heads + h) * vdim + e] =
                  o[((size_t)st * b.n + t) * m.out_ld + (size_t)h * m.vdim + e];
    }
    std::vector<float> s(state_bytes / 4);
    LB_CUDA(cudaMemcpy(s.data(), m.state, state_bytes, cudaMemcpyDeviceToHost));
    for (int st = 0; st < n_streams; ++st)
      for (int h = 0; h < heads; ++h)
        for (int d = 0; d < dim; ++d)
          for (int e = 0; e < vdim; ++e)
            state[(((size_t)st * heads + h) * dim + d) * vdim + e] =
                s[((((size_t)st + slot0) * heads + h) * m.dim + d) * m.vdim + e];
    return LITNICE_B200_OK;
  });
}

int litnice_b200_grouped_attention_host(int32_t engine, const float *rows, const float *q_weight, const float *k_weight,
                                        float eps, int32_t rot_dims, const double *turns, float amplitude, int32_t n_streams,
                                        int32_t p0, int32_t n, int32_t heads, int32_t groups, int32_t dim, int32_t vdim,
                                        float scale, int32_t span_kind, int32_t span_size, float *q_out, float *k_out,
                                        float *out) {
  return diag([&]() {
    if (rows == nullptr || q_weight == nullptr || k_weight == nullptr || q_out == nullptr || k_out == nullptr || out == nullptr ||
        engine < 0 || engine > 2 || n_streams <= 0 || p0 < 0 || n <= 0 || heads <= 0 || groups <= 0 || heads % groups != 0 ||
        dim <= 0 || vdim <= 0 || vdim > 1024 || span_size <= 0 || span_kind < 0 || span_kind > 1 || rot_dims < 0 ||
        rot_dims % 2 != 0 || rot_dims > dim || (rot_dims > 0 && turns == nullptr))
      return LITNICE_B200_EINVAL;
    const Precision type = engine == 0 ? Precision::F32 : Precision::BF16;
    const size_t es = type == Precision::BF16 ? 2 : 4;
    Dev dev;
    ErrWord err;
    GroupedAttention a{};
    a.heads = heads;
    a.groups = groups;
    a.dim = up16(dim);
    a.vdim = up16(vdim);
    if (engine == 2 && !grouped_prefill_supports(a.dim, a.vdim)) return LITNICE_B200_EINVAL;
    a.scale = scale;
    a.span.kind = static_cast<SpanKind>(span_kind);
    a.span.size = span_size;
    const int T = p0 + n, slot0 = 1;
    a.cap = T + 5;
    a.slots = n_streams + slot0;
    a.q_ld = heads * a.dim;
    a.out_ld = heads * a.vdim;
    const int qk = (heads + groups) * a.dim, W = qk + groups * a.vdim, true_qk = (heads + groups) * dim,
              true_w = true_qk + groups * vdim;
    const size_t k_bytes = (size_t)a.slots * a.cap * groups * a.dim * es, v_bytes = (size_t)a.slots * a.cap * groups * a.vdim * es;
    a.k_cache = dev.alloc(k_bytes);
    a.v_cache = dev.alloc(v_bytes);
    LB_CUDA(cudaMemset(a.k_cache, 0x41, k_bytes));  // what earlier sequences may have left in the slots
    LB_CUDA(cudaMemset(a.v_cache, 0x41, v_bytes));
    void *q = dev.alloc((size_t)n_streams * T * a.q_ld * es);
    a.q = q;
    a.out = dev.alloc((size_t)n_streams * n * a.out_ld * es);
    auto weight = [&](const float *w, int count) {
      std::vector<float> wide((size_t)count * a.dim, 0.f);
      for (int c = 0; c < count * dim; ++c) wide[(size_t)(c / dim) * a.dim + c % dim] = w[c];
      return static_cast<float *>(put(dev, wide.data(), 1, count * a.dim, count * a.dim, Precision::F32));
    };
    const float *qw = weight(q_weight, heads), *kw = weight(k_weight, groups);
    Rotation rot;
    rot.dims = rot_dims;
    rot.amplitude = amplitude;
    if (rot_dims > 0) {
      double *t = static_cast<double *>(dev.alloc((size_t)rot_dims / 2 * 8));
      LB_CUDA(cudaMemcpy(t, turns, (size_t)rot_dims / 2 * 8, cudaMemcpyHostToDevice));
      rot.turns = t;
    }
    auto enter = [&](int from, int count) {
      RowBatch b;
      b.streams = n_streams;
      b.slot0 = slot0;
      b.p0 = from;
      b.n = count;
      b.s_cap = T;
      std::vector<float> in((size_t)b.rows() * W, 0.f);
      for (int st = 0; st < n_streams; ++st)
        for (int t = 0; t < count; ++t)
          for (int c = 0; c < true_w; ++c) {
            const int to = c < true_qk ? c / dim * a.dim + c % dim : qk + (c - true_qk) / vdim * a.vdim + (c - true_qk) % vdim;
            in[((size_t)st * count + t) * W + to] = rows[((size_t)st * T + from + t) * true_w + c];
          }
      launch_qk_norm_rotate(put(dev, in.data(), b.rows(), W, W, type), W, qw, kw, eps, dim, rot, a, q, type, b, nullptr);
      return b;
    };
    if (p0 > 0) enter(0, p0);
    const RowBatch b = enter(p0, n);
    if (engine == 2) launch_grouped_prefill(a, b, nullptr, err.dev);
    else launch_grouped_attention_rows(a, type, b, nullptr);
    LB_CUDA(cudaDeviceSynchronize());
    if (err.host->code != DEVERR_NONE) return LITNICE_B200_EDEVICE;
    std::vector<float> wide((size_t)n_streams * n * (a.q_ld > a.out_ld ? a.q_ld : a.out_ld));
    get(q, (long long)n_streams * n, a.q_ld, a.q_ld, type, wide.data());
    for (size_t r = 0; r < (size_t)n_streams * n; ++r)
      for (int c = 0; c < heads * dim; ++c) q_out[r * heads * dim + c] = wide[r * a.q_ld + (size_t)(c / dim) * a.dim + c % dim];
    get(a.out, (long long)n_streams * n, a.out_ld, a.out_ld, type, wide.data());
    for (size_t r = 0; r < (size_t)n_streams * n; ++r)
      for (int c = 0; c < heads * vdim; ++c)
        out[r * heads * vdim + c] = wide[r * a.out_ld + (size_t)(c / vdim) * a.vdim + c % vdim];
    const int kl = groups * a.dim;
    std::vector<float> keys((size_t)a.slots * a.cap * kl);
    get(a.k_cache, (long long)a.slots * a.cap, kl, kl, type, keys.data());
    for (int st = 0; st < n_streams; ++st)
      for (int t = 0; t < T; ++t)
        for (int c = 0; c < groups * dim; ++c)
          k_out[((size_t)st * T + t) * groups * dim + c] =
              keys[((size_t)(st + slot0) * a.cap + t) * kl + (size_t)(c / dim) * a.dim + c % dim];
    return LITNICE_B200_OK;
  });
}

}  // extern "C"
