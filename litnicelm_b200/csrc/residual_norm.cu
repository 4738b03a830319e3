// The norms around a sublayer, one launch for what stands between two products:
//
//   x <- x + y / sqrt(mean(y^2) + eps) * after        (the sublayer's output into the residual stream)
//   h  = x / sqrt(mean(x^2) + eps) * before           (the next sublayer's input)
//
// One CTA per row, the row in registers between the two reductions (four consecutive columns per thread and
// piece); rows of any other width go through a loop over columns that each thread owns. All 32-bit.
#include "model.cuh"

#include <cuda_bf16.h>

namespace lb {

namespace {

constexpr int RN_THREADS = 256;

__device__ __forceinline__ void put4(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void put4(__nv_bfloat16 *p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<const unsigned *>(&a);
  u.y = *reinterpret_cast<const unsigned *>(&b);
  *reinterpret_cast<uint2 *>(p) = u;
}
__device__ __forceinline__ void put(float *p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16 *p, float v) { *p = __float2bfloat16_rn(v); }

// Sum over the CTA, the same bits in every thread.
__device__ __forceinline__ float block_sum(float v, float *part) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
  __syncthreads();
  float s = 0.f;
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) s += part[i];
  return s;
}
__device__ __forceinline__ float4 gain4(const RmsWeight &w, int c) {
  if (w.w == nullptr) return make_float4(w.base, w.base, w.base, w.base);
  const float4 v = *reinterpret_cast<const float4 *>(w.w + c);
  return make_float4(w.base + v.x, w.base + v.y, w.base + v.z, w.base + v.w);
}
__device__ __forceinline__ float squares(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }

template <typename T, int PIECES>
__global__ void __launch_bounds__(RN_THREADS)
residual_norm_kernel(float *x, const float *y, RmsWeight after, T *h, int h_ld, RmsWeight before, int d, float eps) {
  __shared__ float part[2][RN_THREADS / 32];
  pdl_launch_dependents();
  const int c0 = threadIdx.x * 4, step = blockDim.x * 4;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 ga[PIECES], gb[PIECES];  // weights do not depend on the predecessor
#pragma unroll
  for (int i = 0; i < PIECES; ++i) {
    const int c = c0 + i * step;
    ga[i] = y && c < d ? gain4(after, c) : zero;
    gb[i] = h && c < d ? gain4(before, c) : zero;
  }
  pdl_wait();
  float *xr = x + (long long)blockIdx.x * d;
  float4 v[PIECES];
#pragma unroll
  for (int i = 0; i < PIECES; ++i) v[i] = c0 + i * step < d ? *reinterpret_cast<const float4 *>(xr + c0 + i * step) : zero;
  if (y) {
    const float *yr = y + (long long)blockIdx.x * d;
    float4 w[PIECES];
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < PIECES; ++i) {
      w[i] = c0 + i * step < d ? *reinterpret_cast<const float4 *>(yr + c0 + i * step) : zero;
      s += squares(w[i]);
    }
    const float inv = 1.0f / sqrtf(block_sum(s, part[0]) / (float)d + eps);
#pragma unroll
    for (int i = 0; i < PIECES; ++i) {
      v[i].x += w[i].x * inv * ga[i].x;
      v[i].y += w[i].y * inv * ga[i].y;
      v[i].z += w[i].z * inv * ga[i].z;
      v[i].w += w[i].w * inv * ga[i].w;
      if (c0 + i * step < d) put4(xr + c0 + i * step, v[i]);
    }
  }
  if (h == nullptr) return;
  float s = 0.f;
#pragma unroll
  for (int i = 0; i < PIECES; ++i) s += squares(v[i]);
  const float inv = 1.0f / sqrtf(block_sum(s, part[1]) / (float)d + eps);
  T *hr = h + (long long)blockIdx.x * h_ld;
#pragma unroll
  for (int i = 0; i < PIECES; ++i)
    if (c0 + i * step < d)
      put4(hr + c0 + i * step, make_float4(v[i].x * inv * gb[i].x, v[i].y * inv * gb[i].y, v[i].z * inv * gb[i].z,
                                           v[i].w * inv * gb[i].w));
}

template <typename T>
__global__ void __launch_bounds__(RN_THREADS)
residual_norm_any_kernel(float *x, const float *y, RmsWeight after, T *h, int h_ld, RmsWeight before, int d, float eps) {
  __shared__ float part[2][RN_THREADS / 32];
  pdl_launch_dependents();
  pdl_wait();
  float *xr = x + (long long)blockIdx.x * d;
  if (y) {
    const float *yr = y + (long long)blockIdx.x * d;
    float s = 0.f;
    for (int c = threadIdx.x; c < d; c += RN_THREADS) s = fmaf(yr[c], yr[c], s);
    const float inv = 1.0f / sqrtf(block_sum(s, part[0]) / (float)d + eps);
    for (int c = threadIdx.x; c < d; c += RN_THREADS) xr[c] += yr[c] * inv * after.at(c);
  }
  if (h == nullptr) return;
  float s = 0.f;
  for (int c = threadIdx.x; c < d; c += RN_THREADS) s = fmaf(xr[c], xr[c], s);
  const float inv = 1.0f / sqrtf(block_sum(s, part[1]) / (float)d + eps);
  T *hr = h + (long long)blockIdx.x * h_ld;
  for (int c = threadIdx.x; c < d; c += RN_THREADS) put(hr + c, xr[c] * inv * before.at(c));
}

template <typename T>
void launch_t(float *x, const float *y, const RmsWeight &after, T *h, int h_ld, const RmsWeight &before, int d, long long rows,
              float eps, cudaStream_t st) {
  auto go = [&](auto kernel, int threads) {
    launch_pdl(kernel, dim3((unsigned)rows), dim3((unsigned)threads), 0, st, g_pdl_enabled, x, y, after, h, h_ld, before, d,
               eps);
  };
  const int quads = d / 4;
  if (d % 4 != 0 || h_ld % 4 != 0 || quads > 8 * RN_THREADS) return go(residual_norm_any_kernel<T>, RN_THREADS);
  auto threads = [&](int pieces) { return ((quads + pieces - 1) / pieces + 31) / 32 * 32; };
  if (quads <= RN_THREADS) go(residual_norm_kernel<T, 1>, threads(1));
  else if (quads <= 2 * RN_THREADS) go(residual_norm_kernel<T, 2>, threads(2));
  else if (quads <= 4 * RN_THREADS) go(residual_norm_kernel<T, 4>, threads(4));
  else go(residual_norm_kernel<T, 8>, threads(8));
}

}  // namespace

void launch_residual_norm(float *x, const float *y, const RmsWeight &after, void *h, int h_ld, const RmsWeight &before, int d,
                          long long rows, float eps, Precision type, cudaStream_t st) {
  if (type == Precision::BF16) launch_t(x, y, after, static_cast<__nv_bfloat16 *>(h), h_ld, before, d, rows, eps, st);
  else launch_t(x, y, after, static_cast<float *>(h), h_ld, before, d, rows, eps, st);
}

}  // namespace lb
