// Scalar-gain RMS norm and the short causal convolution on a sublayer's input.
//
//   h_t = x_t / sqrt(mean(x_t^2) + eps) * gain          (gain: one number)
//   a_t = h_t + sum_j w[j] * h_(t - taps + 1 + j)        (per channel; zeros before the sequence)
//
// for one or two sublayers that read the same h. The last taps - 1 rows h of a
// stream are its state: history[slot][position % (taps - 1)][d]. A launch covers a
// strip of rows per CTA; rows of the same portion before the strip are recomputed
// from x, rows of earlier portions come from the history. Only a stream's first strip
// touches the history (reads it, then stores the portion's last rows), so no other
// CTA can see it half updated. All arithmetic in 32-bit.
#include "model.cuh"

#include <cuda_bf16.h>

namespace lb {

namespace {

constexpr int CN_THREADS = 256;
constexpr int CN_STRIP = 8;  // rows per CTA (more when taps - 1 is larger)

template <typename T>
__device__ __forceinline__ T from_float(float v);
template <>
__device__ __forceinline__ float from_float<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_float<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

struct ConvPair {
  const float *w[2];
  void *out[2];
  int ld[2];
  int count;
};

// Sum of squares of one row by one warp, 16-byte loads where the row allows them.
__device__ __forceinline__ float warp_inv_rms(const float *row, int d, float eps, int lane) {
  float s = 0.f;
  if ((d & 3) == 0) {
    const float4 *p = reinterpret_cast<const float4 *>(row);
#pragma unroll 4
    for (int c = lane; c < (d >> 2); c += 32) {
      const float4 v = p[c];
      s += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
  } else {
    for (int c = lane; c < d; c += 32) s += row[c] * row[c];
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
  return 1.0f / sqrtf(s / (float)d + eps);
}

// TAPS > 0: that many taps, the window of h kept in registers; 0: any number.
template <typename T, int TAPS>
__global__ void __launch_bounds__(CN_THREADS)
rms_canon_kernel(const float *x, int d, float gain, float eps, int taps_any, float *history,
                 ConvPair cv, int n, int p0_host, const LoopState *state, int slot0, int strip) {
  // (any width and number of taps)
  extern __shared__ float inv[];  // [halo + strip] of this strip, then [halo] of the portion's last rows
  pdl_launch_dependents();
  pdl_wait();
  const int taps = TAPS > 0 ? TAPS : taps_any;
  const int halo = taps - 1;
  const int ring = halo > 0 ? halo : 1;
  const int b = blockIdx.y, t0 = blockIdx.x * strip;
  const int rows = min(strip, n - t0);
  const int p0 = state ? state->s - n : p0_host;
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  const float *xs = x + (long long)b * n * d;
  float *hist = history + (long long)(slot0 + b) * halo * d;
  const bool first = blockIdx.x == 0;
  const int tail0 = max(0, n - halo);  // rows whose h stays behind as the stream's state
  for (int i = wid; i < halo + rows + (first ? n - tail0 : 0); i += CN_THREADS / 32) {
    const int t = i < halo + rows ? t0 - halo + i : tail0 + (i - halo - rows);
    if (t >= 0) {
      const float v = warp_inv_rms(xs + (long long)t * d, d, eps, lane) * gain;
      if (lane == 0) inv[i] = v;
    }
  }
  __syncthreads();
  // h of row t (>= -halo) of the portion, channel c
  auto h_at = [&](int t, int c) -> float {
    if (t >= 0) return xs[(long long)t * d + c] * inv[t - t0 + halo];
    const int p = p0 + t;
    return p >= 0 ? hist[(long long)(p % ring) * d + c] : 0.f;
  };
  for (int c = threadIdx.x; c < d; c += CN_THREADS) {
    if (TAPS > 0) {
      constexpr int TP = TAPS > 0 ? TAPS : 1;
      float w0[TP], w1[TP], win[TP];
#pragma unroll
      for (int j = 0; j < TP; ++j) {
        w0[j] = cv.w[0][(long long)j * d + c];
        w1[j] = cv.count > 1 ? cv.w[1][(long long)j * d + c] : 0.f;
      }
#pragma unroll
      for (int j = 0; j < TP - 1; ++j) win[j + 1] = h_at(t0 - (TP - 1) + j, c);
      for (int t = t0; t < t0 + rows; ++t) {
#pragma unroll
        for (int j = 0; j + 1 < TP; ++j) win[j] = win[j + 1];
        win[TP - 1] = h_at(t, c);
        float a0 = 0.f, a1 = 0.f;
#pragma unroll
        for (int j = 0; j < TP; ++j) {
          a0 = fmaf(w0[j], win[j], a0);
          a1 = fmaf(w1[j], win[j], a1);
        }
        const long long r = (long long)b * n + t;
        static_cast<T *>(cv.out[0])[r * cv.ld[0] + c] = from_float<T>(win[TP - 1] + a0);
        if (cv.count > 1) static_cast<T *>(cv.out[1])[r * cv.ld[1] + c] = from_float<T>(win[TP - 1] + a1);
      }
    } else {
      for (int t = t0; t < t0 + rows; ++t) {
        float a0 = 0.f, a1 = 0.f;
        for (int j = 0; j < taps; ++j) {
          const float h = h_at(t - halo + j, c);
          a0 = fmaf(cv.w[0][(long long)j * d + c], h, a0);
          if (cv.count > 1) a1 = fmaf(cv.w[1][(long long)j * d + c], h, a1);
        }
        const float h = h_at(t, c);
        const long long r = (long long)b * n + t;
        static_cast<T *>(cv.out[0])[r * cv.ld[0] + c] = from_float<T>(h + a0);
        if (cv.count > 1) static_cast<T *>(cv.out[1])[r * cv.ld[1] + c] = from_float<T>(h + a1);
      }
    }
    // The channel's reads of the history are done; its thread alone writes it.
    if (first)
      for (int t = tail0; t < n; ++t)
        hist[(long long)((p0 + t) % ring) * d + c] = xs[(long long)t * d + c] * inv[halo + rows + (t - tail0)];
  }
}

__device__ __forceinline__ void store4(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16 *p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<const unsigned *>(&a);
  u.y = *reinterpret_cast<const unsigned *>(&b);
  *reinterpret_cast<uint2 *>(p) = u;
}
__device__ __forceinline__ float4 fma4(float4 a, float4 b, float4 c) {
  return make_float4(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y), fmaf(a.z, b.z, c.z), fmaf(a.w, b.w, c.w));
}

// The same for rows that fit a CTA's registers, four channels per thread (d % 4 == 0, d <= 4 * blockDim.x):
// the strip's rows, the rows before it and the weights are requested at once, every row of x is read one
// time, and all rows' sums of squares meet in one block reduction. ROWS: rows per strip.
template <typename T, int TAPS, int ROWS, int THREADS>
__global__ void __launch_bounds__(THREADS)
rms_canon_vec_kernel(const float *x, int d, float gain, float eps, float *history, ConvPair cv,
                     int n, int p0_host, const LoopState *state, int slot0) {
  constexpr int HALO = TAPS - 1, RING = HALO > 0 ? HALO : 1, ALL = HALO + ROWS;
  constexpr bool TAIL = ROWS > 1;  // the portion's last rows may lie outside the first strip
  constexpr int SUMS = ALL + (TAIL ? HALO : 0);
  __shared__ float part[32][SUMS];
  __shared__ float inv_s[SUMS];
  pdl_launch_dependents();
  const int c = threadIdx.x * 4;
  const bool in = c < d;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 w[2][TAPS];  // weights do not depend on the predecessor
#pragma unroll
  for (int i = 0; i < 2; ++i)
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
      w[i][j] = in && i < cv.count ? *reinterpret_cast<const float4 *>(cv.w[i] + (long long)j * d + c) : zero;
  pdl_wait();
  const int b = blockIdx.y, t0 = blockIdx.x * ROWS;
  const int rows = min(ROWS, n - t0);
  const int p0 = state ? state->s - n : p0_host;
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  const float *xs = x + (long long)b * n * d + c;
  float *hist = history + (long long)(slot0 + b) * HALO * d + c;
  const bool first = blockIdx.x == 0;
  float4 r[ALL];  // rows t0 - HALO .. t0 + ROWS - 1: x where this portion has it, else the stored h
#pragma unroll
  for (int i = 0; i < ALL; ++i) {
    const int t = t0 - HALO + i;
    r[i] = zero;
    if (in && t < t0 + rows) {
      if (t >= 0) r[i] = *reinterpret_cast<const float4 *>(xs + (long long)t * d);
      else if (p0 + t >= 0) r[i] = *reinterpret_cast<const float4 *>(hist + (long long)((p0 + t) % RING) * d);
    }
  }
  const int tail0 = max(0, n - HALO);
  float4 tail[TAIL && HALO > 0 ? HALO : 1];
  if (TAIL && first) {
#pragma unroll
    for (int i = 0; i < HALO; ++i)
      tail[i] = in && tail0 + i < n ? *reinterpret_cast<const float4 *>(xs + (long long)(tail0 + i) * d) : zero;
  }
#pragma unroll
  for (int i = 0; i < SUMS; ++i) {
    const float4 v = i < ALL ? r[i] : first ? tail[i < ALL ? 0 : i - ALL] : zero;
    float s = v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    if (lane == 0) part[wid][i] = s;
  }
  __syncthreads();
  if (threadIdx.x < SUMS) {
    float s = 0.f;
    for (int q = 0; q < (int)(blockDim.x >> 5); ++q) s += part[q][threadIdx.x];
    inv_s[threadIdx.x] = 1.0f / sqrtf(s / (float)d + eps) * gain;
  }
  __syncthreads();
  if (!in) return;
#pragma unroll
  for (int i = 0; i < ALL; ++i) {
    if (t0 - HALO + i >= 0) {  // stored rows are h already
      const float f = inv_s[i];
      r[i] = make_float4(r[i].x * f, r[i].y * f, r[i].z * f, r[i].w * f);
    }
  }
#pragma unroll
  for (int i = 0; i < ROWS; ++i) {
    if (i >= rows) break;
    float4 a0 = zero, a1 = zero;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      a0 = fma4(w[0][j], r[i + j], a0);
      a1 = fma4(w[1][j], r[i + j], a1);
    }
    const float4 h = r[i + HALO];
    const long long row = (long long)b * n + t0 + i;
    store4(static_cast<T *>(cv.out[0]) + row * cv.ld[0] + c, make_float4(h.x + a0.x, h.y + a0.y, h.z + a0.z, h.w + a0.w));
    if (cv.count > 1)
      store4(static_cast<T *>(cv.out[1]) + row * cv.ld[1] + c, make_float4(h.x + a1.x, h.y + a1.y, h.z + a1.z, h.w + a1.w));
  }
  // The channels' reads of the history are done; their thread alone writes them.
  if (first && HALO > 0) {
    if (TAIL) {
#pragma unroll
      for (int i = 0; i < HALO; ++i) {
        if (tail0 + i >= n) break;
        const float f = inv_s[i + ALL < SUMS ? i + ALL : 0];
        store4(hist + (long long)((p0 + tail0 + i) % RING) * d,
               make_float4(tail[i].x * f, tail[i].y * f, tail[i].z * f, tail[i].w * f));
      }
    } else {
      store4(hist + (long long)(p0 % RING) * d, r[ALL - 1]);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(CN_THREADS)
rms_rows_kernel(const float *x, int d, RmsWeight weight, float eps, const int *rows_list,
                int n_per_stream, T *__restrict__ out, int ld) {
  __shared__ float part[CN_THREADS / 32];
  pdl_launch_dependents();
  pdl_wait();
  const int r = blockIdx.x, lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  const long long src = rows_list ? rows_list[r] : (long long)(r + 1) * n_per_stream - 1;
  const float *row = x + src * d;
  float s = 0.f;
  for (int c = threadIdx.x; c < d; c += CN_THREADS) s = fmaf(row[c], row[c], s);
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
  if (lane == 0) part[wid] = s;
  __syncthreads();
  s = 0.f;
#pragma unroll
  for (int i = 0; i < CN_THREADS / 32; ++i) s += part[i];
  const float inv = 1.0f / sqrtf(s / (float)d + eps);
  for (int c = threadIdx.x; c < d; c += CN_THREADS) out[(long long)r * ld + c] = from_float<T>(row[c] * inv * weight.at(c));
}

template <typename T>
void launch_canon_t(const float *x, int d, float gain, float eps, int taps, float *history, const ConvPair &cv,
                    const RowBatch &b, cudaStream_t st) {
  const int strip = taps - 1 > CN_STRIP ? taps - 1 : CN_STRIP;
  const dim3 grid((unsigned)((b.n + strip - 1) / strip), (unsigned)b.streams);
  const size_t smem = (size_t)(strip + 2 * (taps - 1)) * sizeof(float);
  const bool aligned = (cv.ld[0] & 3) == 0 && (cv.count < 2 || (cv.ld[1] & 3) == 0);
  if ((d & 3) == 0 && d <= 4096 && taps <= 4 && aligned) {
    const unsigned threads = (unsigned)((d / 4 + 31) / 32 * 32);
    auto vec = [&](auto kernel, int rows) {
      launch_pdl(kernel, dim3((unsigned)((b.n + rows - 1) / rows), (unsigned)b.streams), dim3(threads), 0, st, g_pdl_enabled, x,
                 d, gain, eps, history, cv, b.n, b.p0, b.state, b.slot0);
    };
    // rows per strip: one when decoding; else 8, or 4 where the rows are wide (a strip covers at least the
    // taps - 1 rows that the next one reads back to)
    switch (taps * 3 + (b.n == 1 ? 0 : threads <= 512 ? 1 : 2)) {
      case 3: return vec(rms_canon_vec_kernel<T, 1, 1, 1024>, 1);
      case 4: return vec(rms_canon_vec_kernel<T, 1, 8, 512>, 8);
      case 5: return vec(rms_canon_vec_kernel<T, 1, 4, 1024>, 4);
      case 6: return vec(rms_canon_vec_kernel<T, 2, 1, 1024>, 1);
      case 7: return vec(rms_canon_vec_kernel<T, 2, 8, 512>, 8);
      case 8: return vec(rms_canon_vec_kernel<T, 2, 4, 1024>, 4);
      case 9: return vec(rms_canon_vec_kernel<T, 3, 1, 1024>, 1);
      case 10: return vec(rms_canon_vec_kernel<T, 3, 8, 512>, 8);
      case 11: return vec(rms_canon_vec_kernel<T, 3, 4, 1024>, 4);
      case 12: return vec(rms_canon_vec_kernel<T, 4, 1, 1024>, 1);
      case 13: return vec(rms_canon_vec_kernel<T, 4, 8, 512>, 8);
      default: return vec(rms_canon_vec_kernel<T, 4, 4, 1024>, 4);
    }
  }
  auto go = [&](auto kernel) {
    launch_pdl(kernel, grid, dim3(CN_THREADS), smem, st, g_pdl_enabled, x, d, gain, eps, taps, history, cv, b.n, b.p0,
               b.state, b.slot0, strip);
  };
  switch (taps) {
    case 1: go(rms_canon_kernel<T, 1>); break;
    case 2: go(rms_canon_kernel<T, 2>); break;
    case 3: go(rms_canon_kernel<T, 3>); break;
    case 4: go(rms_canon_kernel<T, 4>); break;
    default: go(rms_canon_kernel<T, 0>);
  }
}

}  // namespace

void launch_rms_canon(const float *x, int d, float gain, float eps, int taps, float *history, const CanonConv *conv,
                      int n_conv, Precision type, const RowBatch &b, cudaStream_t st) {
  ConvPair cv{};
  cv.count = n_conv;
  for (int i = 0; i < n_conv; ++i) {
    cv.w[i] = conv[i].w;
    cv.out[i] = conv[i].out;
    cv.ld[i] = conv[i].ld;
  }
  if (type == Precision::BF16) launch_canon_t<__nv_bfloat16>(x, d, gain, eps, taps, history, cv, b, st);
  else launch_canon_t<float>(x, d, gain, eps, taps, history, cv, b, st);
}

void launch_rms_rows(const float *x, int d, const RmsWeight &weight, float eps, const int *rows_dev, int n_rows, int n_per_stream,
                     void *out, int ld, Precision type, cudaStream_t st) {
  if (type == Precision::BF16)
    launch_pdl(rms_rows_kernel<__nv_bfloat16>, dim3((unsigned)n_rows), dim3(CN_THREADS), 0, st, g_pdl_enabled, x, d, weight,
               eps, rows_dev, n_per_stream, static_cast<__nv_bfloat16 *>(out), ld);
  else
    launch_pdl(rms_rows_kernel<float>, dim3((unsigned)n_rows), dim3(CN_THREADS), 0, st, g_pdl_enabled, x, d, weight, eps,
               rows_dev, n_per_stream, static_cast<float *>(out), ld);
}

}  // namespace lb
