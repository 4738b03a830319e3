// Weights of a model folder on their way from the file image in device memory to
// the layouts the kernels read, and the float elementwise step that the 32-bit
// path runs between two products.
#include "activation.cuh"
#include "model.cuh"

#include <cuda_bf16.h>

namespace lb {

namespace {

__device__ __forceinline__ void flag_non_finite(unsigned short bits, DevErr *err) {
  if ((bits & 0x7f80u) == 0x7f80u) {
    err->code = DEVERR_NON_FINITE;
    err->detail = (int)bits;
  }
}

// Tensors start at 2-byte granularity inside a file image, so loads are 16-bit.
__global__ void pack_bf16_kernel(const unsigned short *__restrict__ src, long long rows, int cols,
                                 unsigned short *__restrict__ dst, long long ld, DevErr *err) {
  const long long total = rows * cols;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / cols;
    const unsigned short v = src[i];
    flag_non_finite(v, err);
    dst[r * ld + (i - r * cols)] = v;
  }
}

__global__ void expand_f32_kernel(const unsigned short *__restrict__ src, long long rows, int cols,
                                  float *__restrict__ dst, long long ld, int transpose, DevErr *err) {
  const long long total = rows * cols;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    const long long r = i / cols, c = i - r * cols;
    const unsigned short v = src[i];
    flag_non_finite(v, err);
    dst[transpose ? c * ld + r : r * ld + c] = __uint_as_float((unsigned)v << 16);
  }
}

template <typename T>
__device__ __forceinline__ T from_bits(unsigned short v);
template <>
__device__ __forceinline__ unsigned short from_bits<unsigned short>(unsigned short v) { return v; }
template <>
__device__ __forceinline__ float from_bits<float>(unsigned short v) { return __uint_as_float((unsigned)v << 16); }

template <typename T>
__global__ void place_kernel(const unsigned short *__restrict__ src, long long rows, int cols, T *__restrict__ dst,
                             WeightPlace at, DevErr *err) {
  const long long total = rows * cols;
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
    long long r = i / cols, c = i - r * cols;
    const unsigned short v = src[i];
    flag_non_finite(v, err);
    if (at.row_group > 0) r = r / at.row_group * at.row_pad + r % at.row_group;
    if (at.col_group > 0) c = c / at.col_group * at.col_pad + c % at.col_group;
    dst[at.offset + r * at.row_stride + c * at.col_stride] = from_bits<T>(v);
  }
}

// x <- act(x) (* factor).
__global__ void activation_f32_kernel(float *x, const float *factor, long long count, int act) {
  pdl_launch_dependents();
  pdl_wait();
  for (long long i = blockIdx.x * (long long)blockDim.x + threadIdx.x; i < count; i += (long long)gridDim.x * blockDim.x) {
    const float z = activate(x[i], act);
    x[i] = factor ? z * factor[i] : z;
  }
}

unsigned blocks_for(long long count) {
  const long long b = (count + 255) / 256;
  return (unsigned)(b < 1 ? 1 : b > 4736 ? 4736 : b);
}

}  // namespace

void launch_pack_bf16(const void *src, long long rows, int cols, void *dst, long long ld, cudaStream_t st, DevErr *err) {
  pack_bf16_kernel<<<blocks_for(rows * cols), 256, 0, st>>>(static_cast<const unsigned short *>(src), rows, cols,
                                                            static_cast<unsigned short *>(dst), ld, err);
  LB_LAUNCH_CHECK();
}

void launch_expand_f32(const void *src, long long rows, int cols, float *dst, long long ld, bool transpose,
                       cudaStream_t st, DevErr *err) {
  expand_f32_kernel<<<blocks_for(rows * cols), 256, 0, st>>>(static_cast<const unsigned short *>(src), rows, cols, dst,
                                                             ld, transpose ? 1 : 0, err);
  LB_LAUNCH_CHECK();
}

void launch_place(const void *src, long long rows, int cols, void *dst, Precision type, const WeightPlace &at,
                  cudaStream_t st, DevErr *err) {
  const unsigned short *from = static_cast<const unsigned short *>(src);
  if (type == Precision::BF16)
    place_kernel<unsigned short><<<blocks_for(rows * cols), 256, 0, st>>>(from, rows, cols, static_cast<unsigned short *>(dst),
                                                                          at, err);
  else
    place_kernel<float><<<blocks_for(rows * cols), 256, 0, st>>>(from, rows, cols, static_cast<float *>(dst), at, err);
  LB_LAUNCH_CHECK();
}

void launch_activation_f32(float *x, const float *factor, long long count, Activation act, cudaStream_t st) {
  launch_pdl(activation_f32_kernel, dim3(blocks_for(count)), dim3(256), 0, st, g_pdl_enabled, x, factor, count, (int)act);
}

}  // namespace lb
