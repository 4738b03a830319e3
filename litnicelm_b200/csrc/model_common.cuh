// What the registered decoder designs share on the host: device buffers that grow, slot
// buffers, and the matrix products of both precisions.
#pragma once

#include <utility>

#include "gemm_tc.cuh"
#include "model.cuh"

namespace lb {

inline int up8(int v) { return (v + 7) & ~7; }
inline int up16(int v) { return (v + 15) & ~15; }

struct DevBuf {
  void *p = nullptr;
  size_t bytes = 0;
  DevBuf() = default;
  DevBuf(const DevBuf &) = delete;
  DevBuf &operator=(const DevBuf &) = delete;
  DevBuf(DevBuf &&o) noexcept : p(o.p), bytes(o.bytes) {
    o.p = nullptr;
    o.bytes = 0;
  }
  ~DevBuf() {
    if (p) cudaFree(p);
  }
  // At least `need` bytes, zeroed when new; true when the buffer moved (its content is gone).
  bool ensure(size_t need, cudaStream_t st) {
    if (need <= bytes) return false;
    if (p) {
      LB_CUDA(cudaStreamSynchronize(st));
      cudaFree(p);
      p = nullptr;
      bytes = 0;
    }
    need = (need + 255) & ~(size_t)255;
    if (cudaMalloc(&p, need) != cudaSuccess) {
      p = nullptr;
      (void)cudaGetLastError();
      throw std::bad_alloc();
    }
    bytes = need;
    LB_CUDA(cudaMemsetAsync(p, 0, need, st));
    return true;
  }
  // A [slots][pitch] buffer to more or longer slots, what it holds kept.
  void grow(size_t old_bytes, int old_slots, size_t old_pitch, int slots, size_t pitch, cudaStream_t st) {
    DevBuf next;
    next.ensure(pitch * slots, st);
    if (p && old_bytes > 0 && old_slots > 0)
      LB_CUDA(cudaMemcpy2DAsync(next.p, pitch, p, old_pitch, old_bytes, (size_t)old_slots, cudaMemcpyDeviceToDevice, st));
    LB_CUDA(cudaStreamSynchronize(st));
    std::swap(p, next.p);
    std::swap(bytes, next.bytes);
  }
  float *f() const { return static_cast<float *>(p); }
};

inline MatView dense_view(const float *p, long long rows, long long cols) {
  MatView v{};
  v.data = reinterpret_cast<char *>(const_cast<float *>(p));
  v.batch = 1;
  v.rows = rows;
  v.cols = cols;
  v.rs = cols * 4;
  v.cs = 4;
  return v;
}

// One or two products on bfloat16 operands by the kernel that suits their rows; returns the kernels launched.
inline int products_bf16(const Bf16Product *p, int count, int m, cudaStream_t st, DevErr *err) {
  if (m <= FEW_ROWS_MAX) {
    launch_few_row_bf16(p, count, m, st);
    return 1;
  }
  for (int i = 0; i < count; ++i) launch_gemm_bf16(p[i], m, st, err);
  return count;
}

// out[m, n] = a[m, k] w[k, n] (+ residual) on the float products; scratch: gemv_scratch_floats(8, n, k) floats.
inline int product_f32(const float *a, int m, int k, const float *w, int n, const float *residual, float *out,
                       float *scratch, cudaStream_t st, DevErr *err) {
  if (m <= 8) return launch_gemv(a, m, w, k, n, nullptr, out, scratch, st, err, residual);
  GemmEpilogue ep;
  ep.residual = residual;
  launch_gemm_simt(dense_view(a, m, k), dense_view(w, k, n), dense_view(out, m, n), m, n, k, ep, st);
  return 1;
}

}  // namespace lb
