// The gated delta rule token by token, and what surrounds it: the short causal convolution with SiLU on
// queries, keys and values, and the gated norm of each head's output.
//
//   delta_conv_kernel   convolution of a portion's rows, its last inputs kept as the slot's history
//   delta_step_kernel   the recurrence, state in registers: CTA = one head (and 32 to 128 of its value columns)
//                       of one stream, warps share the state's rows. FUSED (one new row per stream): convolution,
//                       recurrence, norm and gate in one launch; otherwise any number of rows in order
//   delta_norm_kernel   norm and gate of rows whose outputs lie in memory
//
// With the unscaled vectors k', q' and r = 1 / |k'|, r' = dim^-1/2 / |q'| (norms of what the matrix products
// read), one pass over the state gives both sums a token needs:
//   a = S^T k',  c = S^T q';  u = beta (v - g r a);  o = g r' c + r r' (k' . q') u;  S <- g S + r k' u^T
// which is the rule's order (decay, write, then read) with the read taken before the write is stored.
// All arithmetic 32-bit; the history is stored by position modulo the number of taps: a single new row
// never overwrites an input that another CTA still reads.
#include "delta.cuh"
#include "tc_ptx.cuh"

namespace lb {

namespace {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float4 load4(const float *p) { return *reinterpret_cast<const float4 *>(p); }
__device__ __forceinline__ float4 load4(const bf16 *p) {
  const uint2 u = *reinterpret_cast<const uint2 *>(p);
  return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16),
                     __uint_as_float(u.y & 0xffff0000u));
}
__device__ __forceinline__ void store4(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void store4(bf16 *p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<const unsigned *>(&a);
  u.y = *reinterpret_cast<const unsigned *>(&b);
  *reinterpret_cast<uint2 *>(p) = u;
}
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// ---- convolution -----------------------------------------------------------------

constexpr int DC_THREADS = 128;
constexpr int DC_STRIP = 32;  // rows per CTA (more when taps - 1 is larger)

// 16 bytes of a row.
template <typename T>
struct Wide;
template <>
struct Wide<float> {
  static constexpr int N = 4;
  static __device__ __forceinline__ void unpack(uint4 u, float (&f)[4]) {
    f[0] = __uint_as_float(u.x);
    f[1] = __uint_as_float(u.y);
    f[2] = __uint_as_float(u.z);
    f[3] = __uint_as_float(u.w);
  }
  static __device__ __forceinline__ void store(float *p, const float (&f)[4]) {
    *reinterpret_cast<float4 *>(p) = make_float4(f[0], f[1], f[2], f[3]);
  }
  static __device__ __forceinline__ float silu(float z) { return silu_f32(z); }
};
template <>
struct Wide<bf16> {
  static constexpr int N = 8;
  static __device__ __forceinline__ void unpack(uint4 u, float (&f)[8]) {
    const unsigned w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      f[2 * i] = __uint_as_float(w[i] << 16);
      f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
  }
  static __device__ __forceinline__ void store(bf16 *p, const float (&f)[8]) {
    unsigned w[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const __nv_bfloat162 v = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
      w[i] = *reinterpret_cast<const unsigned *>(&v);
    }
    *reinterpret_cast<uint4 *>(p) = make_uint4(w[0], w[1], w[2], w[3]);
  }
  static __device__ __forceinline__ float silu(float z) { return silu_fast(z); }
};

__device__ __forceinline__ uint4 load16(const void *p) { return *reinterpret_cast<const uint4 *>(p); }

// TAPS > 0: that many taps, the window of inputs in registers; 0: any number. 16 bytes of channels per thread.
template <typename T, int TAPS>
__global__ void __launch_bounds__(DC_THREADS)
delta_conv_kernel(const T *in, int in_ld, const float *__restrict__ w, int taps_any, int channels, T *history, T *out,
                  DeltaRows g, int strip) {
  constexpr int N = Wide<T>::N, TP = TAPS > 0 ? TAPS : 1;
  pdl_launch_dependents();
  const int taps = TAPS > 0 ? TAPS : taps_any;
  const int c = (blockIdx.z * DC_THREADS + threadIdx.x) * N;
  const bool mine = c < channels;
  float wt[TP][N];
  auto weights = [&](int j, float (&f)[N]) {
#pragma unroll
    for (int i = 0; i < N; i += 4) {
      const float4 v = load4(w + (long long)j * channels + c + i);
      f[i] = v.x;
      f[i + 1] = v.y;
      f[i + 2] = v.z;
      f[i + 3] = v.w;
    }
  };
  if (TAPS > 0 && mine) {
#pragma unroll
    for (int j = 0; j < TP; ++j) weights(j, wt[j]);
  }
  pdl_wait();
  if (!mine) return;
  const int b = blockIdx.y, t0 = blockIdx.x * strip, t1 = min(g.n, t0 + strip);
  const int p0 = g.first_position();
  const T *x = in + (long long)b * g.n * in_ld + c;
  T *hist = history + (long long)(g.slot0 + b) * taps * channels + c;
  T *o = out + (long long)b * g.n * channels + c;
  auto input = [&](int t, float (&f)[N]) {
    const int p = p0 + t;
    if (t >= 0) {
      Wide<T>::unpack(load16(x + (long long)t * in_ld), f);
    } else if (p >= 0) {
      Wide<T>::unpack(load16(hist + (long long)(p % taps) * channels), f);
    } else {
#pragma unroll
      for (int i = 0; i < N; ++i) f[i] = 0.f;
    }
  };
  if (TAPS > 0) {
    float win[TP][N];
#pragma unroll
    for (int j = 0; j < TP - 1; ++j) input(t0 - (TP - 1) + j, win[j + 1]);
    constexpr int AHEAD = 8;  // rows requested together
    for (int ta = t0; ta < t1; ta += AHEAD) {
      uint4 raw[AHEAD];
#pragma unroll
      for (int k = 0; k < AHEAD; ++k) raw[k] = load16(x + (long long)min(ta + k, t1 - 1) * in_ld);
#pragma unroll
      for (int k = 0; k < AHEAD; ++k) {
        if (ta + k >= t1) break;
#pragma unroll
        for (int j = 0; j + 1 < TP; ++j)
#pragma unroll
          for (int i = 0; i < N; ++i) win[j][i] = win[j + 1][i];
        Wide<T>::unpack(raw[k], win[TP - 1]);
        float y[N];
#pragma unroll
        for (int i = 0; i < N; ++i) {
          float a = 0.f;
#pragma unroll
          for (int j = 0; j < TP; ++j) a = fmaf(wt[j][i], win[j][i], a);
          y[i] = Wide<T>::silu(a);
        }
        Wide<T>::store(o + (long long)(ta + k) * channels, y);
      }
    }
  } else {
    for (int t = t0; t < t1; ++t) {
      float y[N] = {};
      for (int j = 0; j < taps; ++j) {
        float f[N], v[N];
        weights(j, f);
        input(t - taps + 1 + j, v);
#pragma unroll
        for (int i = 0; i < N; ++i) y[i] = fmaf(f[i], v[i], y[i]);
      }
#pragma unroll
      for (int i = 0; i < N; ++i) y[i] = Wide<T>::silu(y[i]);
      Wide<T>::store(o + (long long)t * channels, y);
    }
  }
  // Only a stream's first strip reads the history, and this thread alone these channels of it.
  if (blockIdx.x == 0)
    for (int t = max(0, g.n - taps + 1); t < g.n; ++t)
      *reinterpret_cast<uint4 *>(hist + (long long)((p0 + t) % taps) * channels) = load16(x + (long long)t * in_ld);
}

// ---- recurrence --------------------------------------------------------------------

struct StepArgs {
  int heads, groups, dim, vdim, taps;
  float q_scale, count, eps;  // dim^-1/2, value columns the norm counts
  const float *conv, *a_log, *dt_bias, *norm;
  float *state;
  const float *ba;
  int ba_ld, in_ld, out_ld;
  long long rows_ld;  // of the convolved rows
};

// VPT neighbouring floats of a state row.
template <int VPT>
__device__ __forceinline__ void load_cols(const float *p, bool ok, float (&s)[VPT]) {
  if constexpr (VPT == 4) {
    const float4 v = ok ? *reinterpret_cast<const float4 *>(p) : make_float4(0.f, 0.f, 0.f, 0.f);
    s[0] = v.x;
    s[1] = v.y;
    s[2] = v.z;
    s[3] = v.w;
  } else if constexpr (VPT == 2) {
    const float2 v = ok ? *reinterpret_cast<const float2 *>(p) : make_float2(0.f, 0.f);
    s[0] = v.x;
    s[1] = v.y;
  } else {
    s[0] = ok ? *p : 0.f;
  }
}
template <int VPT>
__device__ __forceinline__ void store_cols(float *p, const float (&s)[VPT]) {
  if constexpr (VPT == 4) *reinterpret_cast<float4 *>(p) = make_float4(s[0], s[1], s[2], s[3]);
  else if constexpr (VPT == 2) *reinterpret_cast<float2 *>(p) = make_float2(s[0], s[1]);
  else *p = s[0];
}

// WARPS warps share the state's rows, DPW each; a lane holds VPT value columns. FUSED: the CTAs of a head are a
// cluster (one CTA: none); the squares of its outputs meet in shared memory while each stores its part of the state.
template <typename T, int WARPS, int DPW, int VPT, bool FUSED>
__global__ void __launch_bounds__(WARPS * 32, 512 / (WARPS * 32))
delta_step_kernel(StepArgs a, const T *in, T *history, float *o_rows, T *out, DeltaRows g) {
  constexpr int THREADS = WARPS * 32, VT = 32 * VPT, DIMS = WARPS * DPW;
  constexpr int FILL = (2 * DIMS + VT + THREADS - 1) / THREADS;
  __shared__ __align__(16) float vec[2][2 * DIMS + VT];  // q', k', v of a token
  __shared__ __align__(16) float red[WARPS][2][VT];
  __shared__ float squares;
  pdl_launch_dependents();
  const int tid = threadIdx.x, lane = tid & 31, wid = tid >> 5;
  const int tiles = (a.vdim + VT - 1) / VT;
  const int h = blockIdx.x / tiles, vt = (blockIdx.x - h * tiles) * VT, b = blockIdx.y;
  const int grp = h / (a.heads / a.groups);
  const int v0 = vt + lane * VPT, d0 = wid * DPW;
  const bool v_in = v0 < a.vdim;
  float *S = a.state + ((long long)(g.slot0 + b) * a.heads + h) * a.dim * a.vdim;
  if (v_in && lane % (32 / VPT) == 0) {  // towards L2 while the predecessor ends
#pragma unroll
    for (int i = 0; i < DPW; ++i)
      if (d0 + i < a.dim) asm volatile("prefetch.global.L2 [%0];" ::"l"(S + (long long)(d0 + i) * a.vdim + v0));
  }
  const float a_exp_log = a.a_log[h], bias = a.dt_bias[h];
  pdl_wait();
  float s[DPW][VPT];
#pragma unroll
  for (int i = 0; i < DPW; ++i) {
    const float *row = S + (long long)(d0 + i) * a.vdim + v0;
    load_cols(row, v_in && d0 + i < a.dim, s[i]);
  }
  const int p0 = g.first_position();  // asked for behind the state, whose loads need not wait for it
  if (p0 == 0) {  // a new sequence
#pragma unroll
    for (int i = 0; i < DPW; ++i)
#pragma unroll
      for (int j = 0; j < VPT; ++j) s[i][j] = 0.f;
  }
  // channel of entry e of a token's vectors, or -1 for padding
  auto channel = [&](int e) -> int {
    if (e < DIMS) return e < a.dim ? grp * a.dim + e : -1;
    if (e < 2 * DIMS) return e - DIMS < a.dim ? (a.groups + grp) * a.dim + e - DIMS : -1;
    const int v = vt + e - 2 * DIMS;
    return e < 2 * DIMS + VT && v < a.vdim ? 2 * a.groups * a.dim + h * a.vdim + v : -1;
  };
  const int channels = 2 * a.groups * a.dim + a.heads * a.vdim;
  float next[FILL], next_b, next_a;
  auto fetch = [&](int t) {
    const long long r = (long long)b * g.n + t;
#pragma unroll
    for (int i = 0; i < FILL; ++i) {
      const int c = channel(tid + i * THREADS);
      next[i] = 0.f;
      if (c < 0) continue;
      if constexpr (FUSED) {  // t == 0: the convolution of the one new row
        T *hist = history + (long long)(g.slot0 + b) * a.taps * channels + c;
        const T x = in[r * a.in_ld + c];
        float y = 0.f;
        for (int j = 0; j + 1 < a.taps; ++j) {
          const int p = p0 - a.taps + 1 + j;
          if (p >= 0) y = fmaf(a.conv[(long long)j * channels + c], to_f(hist[(long long)(p % a.taps) * channels]), y);
        }
        y = fmaf(a.conv[(long long)(a.taps - 1) * channels + c], to_f(x), y);
        next[i] = to_f(from_f<T>(Wide<T>::silu(y)));
        if (tid + i * THREADS >= 2 * DIMS || (vt == 0 && h % (a.heads / a.groups) == 0)) hist[(long long)(p0 % a.taps) * channels] = x;
      } else {
        next[i] = to_f(in[r * a.rows_ld + c]);
      }
    }
    next_b = a.ba[r * a.ba_ld + h];
    next_a = a.ba[r * a.ba_ld + a.heads + h];
  };
  fetch(0);
  for (int t = 0; t < g.n; ++t) {
    float *q = vec[t & 1], *k = q + DIMS, *v = k + DIMS;
#pragma unroll
    for (int i = 0; i < FILL; ++i)
      if (tid + i * THREADS < 2 * DIMS + VT) q[tid + i * THREADS] = next[i];
    const float beta = sigmoid_f32(next_b), decay = expf(delta_log_decay(next_a, a_exp_log, bias));
    if (!FUSED && t + 1 < g.n) fetch(t + 1);
    __syncthreads();
    float qq = 0.f, kk = 0.f, kq = 0.f;
    for (int d = lane; d < DIMS; d += 32) {
      qq = fmaf(q[d], q[d], qq);
      kk = fmaf(k[d], k[d], kk);
      kq = fmaf(k[d], q[d], kq);
    }
    float sa[VPT] = {}, sq[VPT] = {};
#pragma unroll
    for (int i = 0; i < DPW; ++i) {
      const float kd = k[d0 + i], qd = q[d0 + i];
#pragma unroll
      for (int j = 0; j < VPT; ++j) {
        sa[j] = fmaf(kd, s[i][j], sa[j]);
        sq[j] = fmaf(qd, s[i][j], sq[j]);
      }
    }
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
      red[wid][0][lane * VPT + j] = sa[j];
      red[wid][1][lane * VPT + j] = sq[j];
    }
    const float rk = 1.0f / sqrtf(warp_sum(kk) + DELTA_UNIT_EPS);
    const float rq = a.q_scale / sqrtf(warp_sum(qq) + DELTA_UNIT_EPS);
    kq = warp_sum(kq) * rk * rq;
    __syncthreads();
    float u[VPT];
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
      float sum = 0.f;
#pragma unroll
      for (int w = 0; w < WARPS; ++w) sum += red[w][0][lane * VPT + j];
      u[j] = beta * (v[lane * VPT + j] - decay * rk * sum);
    }
    float o[VPT];
    if (wid == 0) {
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < VPT; ++j) {
        float sum = 0.f;
#pragma unroll
        for (int w = 0; w < WARPS; ++w) sum += red[w][1][lane * VPT + j];
        o[j] = decay * rq * sum + kq * u[j];
        ss = fmaf(o[j], o[j], ss);
      }
      if constexpr (FUSED) {  // padding columns are zeros
        ss = warp_sum(ss);
        if (lane == 0) squares = ss;
      } else if (v_in) {
        const long long r = (long long)b * g.n + t;
#pragma unroll
        for (int j = 0; j < VPT; ++j) o_rows[(r * a.heads + h) * a.vdim + v0 + j] = o[j];
      }
    }
    if (FUSED && tiles > 1) {
      __syncwarp();
      asm volatile("barrier.cluster.arrive.release.aligned;" ::: "memory");
    }
#pragma unroll
    for (int i = 0; i < DPW; ++i) {
      const float kd = k[d0 + i] * rk;
#pragma unroll
      for (int j = 0; j < VPT; ++j) s[i][j] = fmaf(kd, u[j], decay * s[i][j]);
    }
    if constexpr (FUSED) {
#pragma unroll
      for (int i = 0; i < DPW; ++i)
        if (v_in && d0 + i < a.dim) store_cols(S + (long long)(d0 + i) * a.vdim + v0, s[i]);
      if (tiles > 1) {
        __syncwarp();
        cluster_wait();
      }
      if (wid == 0) {
        __syncwarp();
        float ss = tiles == 1 ? squares : 0.f;
        if (tiles > 1)
          for (int i = 0; i < tiles; ++i) ss += ld_cluster_f32(cluster_map(smem_u32(&squares), (unsigned)i));
        const float inv = 1.0f / sqrtf(ss / a.count + a.eps);
        const T *gate = in + (long long)b * a.in_ld + channels + h * a.vdim;
        T *y = out + (long long)b * a.out_ld + h * a.vdim;
        if (v_in) {
#pragma unroll
          for (int j = 0; j < VPT; ++j)
            y[v0 + j] = from_f<T>(o[j] * inv * a.norm[v0 + j] * Wide<T>::silu(to_f(gate[v0 + j])));
        }
      }
      if (tiles > 1) {  // a CTA's shared memory stays until every other has read it
        __syncwarp();
        cluster_sync_all();
      }
      return;
    }
  }
#pragma unroll
  for (int i = 0; i < DPW; ++i)
    if (v_in && d0 + i < a.dim) store_cols(S + (long long)(d0 + i) * a.vdim + v0, s[i]);
}

// One warp per row and head.
template <typename T>
__global__ void __launch_bounds__(256)
delta_norm_kernel(const float *o_rows, const T *gate, int in_ld, const float *__restrict__ norm, float count, float eps,
                  int heads, int vdim, long long total, T *out, int out_ld) {
  pdl_launch_dependents();
  pdl_wait();
  const long long i = (long long)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (i >= total) return;
  const int lane = threadIdx.x & 31;
  const long long r = i / heads;
  const int h = (int)(i - r * heads);
  const float *o = o_rows + i * vdim;
  float s = 0.f;
  for (int c = lane * 4; c < vdim; c += 128) {
    const float4 v = load4(o + c);
    s += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  const float inv = 1.0f / sqrtf(warp_sum(s) / count + eps);
  for (int c = lane * 4; c < vdim; c += 128) {
    const float4 v = load4(o + c), w = load4(norm + c), z = load4(gate + r * in_ld + h * vdim + c);
    store4(out + r * out_ld + h * vdim + c,
           make_float4(v.x * inv * w.x * silu_f32(z.x), v.y * inv * w.y * silu_f32(z.y), v.z * inv * w.z * silu_f32(z.z),
                       v.w * inv * w.w * silu_f32(z.w)));
  }
}

struct Scratch {
  size_t conv, o, chunk;
};
Scratch scratch_parts(const DeltaMixer &m, long long rows, int streams, Precision type) {
  const size_t es = type == Precision::BF16 ? 2 : 4;
  auto round = [](size_t n) { return (n + 255) & ~(size_t)255; };
  return {round((size_t)rows * m.conv_channels() * es), round((size_t)rows * m.heads * m.vdim * 4),
          type == Precision::BF16 && delta_chunk_supports(m) ? delta_chunk_bytes(m, rows, streams) : 0};
}

constexpr int DELTA_CHUNK_ROWS = 17;  // portions of so many rows per stream and more take the chunked form

template <typename T>
int launch_t(const DeltaMixer &m, void *scratch, Precision type, const RowBatch &b, cudaStream_t st, DevErr *err) {
  const Scratch part = scratch_parts(m, b.rows(), b.streams, type);
  char *at = static_cast<char *>(scratch);
  T *conv = reinterpret_cast<T *>(at);
  float *o = reinterpret_cast<float *>(at + part.conv);
  const T *in = static_cast<const T *>(m.in);
  T *out = static_cast<T *>(m.out);
  const DeltaRows g{b.n, b.p0, b.slot0, b.state};
  StepArgs a{};
  a.heads = m.heads;
  a.groups = m.groups;
  a.dim = m.dim;
  a.vdim = m.vdim;
  a.taps = m.taps;
  a.q_scale = 1.0f / sqrtf((float)m.true_dim);
  a.count = (float)m.true_vdim;
  a.eps = m.eps;
  a.conv = m.conv;
  a.a_log = m.a_log;
  a.dt_bias = m.dt_bias;
  a.norm = m.norm;
  a.state = m.state;
  a.ba = m.ba;
  a.ba_ld = m.ba_ld;
  a.in_ld = m.in_ld;
  a.out_ld = m.out_ld;
  a.rows_ld = m.conv_channels();
  auto step = [&](auto kernel, int threads, int vt, const T *src, bool cluster) {
    const int tiles = (m.vdim + vt - 1) / vt;
    launch_pdl_cluster_x(kernel, dim3((unsigned)(m.heads * tiles), (unsigned)b.streams), dim3((unsigned)threads), 0, st,
                         g_pdl_enabled, cluster ? (unsigned)tiles : 1u, a, src, static_cast<T *>(m.history), o, out, g);
  };
  if (b.n == 1 && m.dim <= 256 && m.vdim <= 256) {
    // the fewest value columns per lane that let one CTA hold a head: splitting a head further gained nothing at any size
    auto fused = [&](auto one, auto two, auto four, int threads) {
      if (m.vdim <= 32) step(one, threads, 32, in, true);
      else if (m.vdim <= 64) step(two, threads, 64, in, true);
      else step(four, threads, 128, in, true);
    };
    if (m.dim <= 64)
      fused(delta_step_kernel<T, 8, 8, 1, true>, delta_step_kernel<T, 8, 8, 2, true>, delta_step_kernel<T, 8, 8, 4, true>, 256);
    else if (m.dim <= 128)
      fused(delta_step_kernel<T, 8, 16, 1, true>, delta_step_kernel<T, 8, 16, 2, true>, delta_step_kernel<T, 8, 16, 4, true>, 256);
    else
      fused(delta_step_kernel<T, 16, 16, 1, true>, delta_step_kernel<T, 16, 16, 2, true>, delta_step_kernel<T, 16, 16, 4, true>,
            512);
    return 1;
  }
  const int strip = m.taps - 1 > DC_STRIP ? m.taps - 1 : DC_STRIP, channels = m.conv_channels();
  auto convolve = [&](auto kernel) {
    launch_pdl(kernel, dim3((unsigned)((b.n + strip - 1) / strip), (unsigned)b.streams,
                            (unsigned)((channels / Wide<T>::N + DC_THREADS - 1) / DC_THREADS)),
               dim3(DC_THREADS), 0, st, g_pdl_enabled, in, m.in_ld, m.conv, m.taps, channels, static_cast<T *>(m.history), conv, g,
               strip);
  };
  switch (m.taps) {
    case 1: convolve(delta_conv_kernel<T, 1>); break;
    case 2: convolve(delta_conv_kernel<T, 2>); break;
    case 3: convolve(delta_conv_kernel<T, 3>); break;
    case 4: convolve(delta_conv_kernel<T, 4>); break;
    default: convolve(delta_conv_kernel<T, 0>);
  }
  int launches = 1;
  if (type == Precision::BF16 && b.n >= DELTA_CHUNK_ROWS && delta_chunk_supports(m)) {
    bool normed = false;
    launches += launch_delta_chunks(m, conv, o, at + part.conv + part.o, b, &normed, st, err);
    if (normed) return launches;
  } else {
    const T *src = conv;
    if (m.dim <= 64) step(delta_step_kernel<T, 8, 8, 4, false>, 256, 128, src, false);
    else if (m.dim <= 128) step(delta_step_kernel<T, 8, 16, 4, false>, 256, 128, src, false);
    else if (m.dim <= 256) step(delta_step_kernel<T, 16, 16, 4, false>, 512, 128, src, false);
    else step(delta_step_kernel<T, 16, 32, 2, false>, 512, 64, src, false);
    ++launches;
  }
  const long long total = b.rows() * m.heads;
  launch_pdl(delta_norm_kernel<T>, dim3((unsigned)((total + 7) / 8)), dim3(256), 0, st, g_pdl_enabled, (const float *)o,
             in + channels, m.in_ld, m.norm, a.count, m.eps, m.heads, m.vdim, total, out, m.out_ld);
  return launches + 1;
}

}  // namespace

bool delta_supports(int dim, int vdim) { return dim % 16 == 0 && vdim % 16 == 0 && dim >= 16 && vdim >= 16 && dim <= 512; }

size_t delta_scratch_bytes(const DeltaMixer &m, long long rows, int streams, Precision type) {
  const Scratch p = scratch_parts(m, rows, streams, type);
  return p.conv + p.o + p.chunk;
}

int launch_delta(const DeltaMixer &m, void *scratch, Precision type, const RowBatch &b, cudaStream_t st, DevErr *err) {
  return type == Precision::BF16 ? launch_t<bf16>(m, scratch, type, b, st, err) : launch_t<float>(m, scratch, type, b, st, err);
}

}  // namespace lb
