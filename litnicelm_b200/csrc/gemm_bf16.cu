// Matrix products on bfloat16 operands for sm_100a (tcgen05 + TMEM + TMA): C[m, n] = A[m, k] W[n, k]^T
// with 32-bit accumulation. The many-row counterpart of few_row_bf16.cu.
//
// Persistent kernel, one CTA per SM, tiles of 128 x BN taken round robin:
//   warp 0      one lane issues the TMA loads of the A and W tiles (64 k per stage, 128-byte swizzle)
//   warp 1      owns tensor memory (two accumulators of BN columns); one lane issues tcgen05.mma
//   warps 2-5   read a finished accumulator and store the tile while the next one is multiplied:
//               32 columns at a time through a padded shared-memory patch, so that global reads and
//               writes are whole rows of 128 bytes
// Rows and columns outside the operands load as zeros (k need not be a multiple of 64) and are not
// stored. Every mbarrier wait is bounded; a wait that runs out sets the error word and ends the kernel
// after its copies have landed and tensor memory is freed. No clusters, no multicast.
#include "activation.cuh"
#include "model.cuh"
#include "gemm_tc.cuh"
#include "tc_ptx.cuh"

#include <cuda_bf16.h>

#include <mutex>

namespace lb {

namespace {

typedef __nv_bfloat16 bf16;

constexpr int GB_THREADS = 192;
constexpr int GB_PATCH_LD = 36;  // floats per row of a warp's staging patch
constexpr int GB_PATCH = 32 * GB_PATCH_LD * 4;
constexpr int GB_GROUP = 16;     // row tiles that share a sweep over the columns (W tiles stay in L2)

template <int BN>
struct GbSmem {
  static constexpr int STAGES = BN == 256 ? 4 : BN == 128 ? 5 : 6;
  static constexpr int A_BYTES = TC_BM * 128;
  static constexpr int B_BYTES = BN * 128;
  static constexpr int STAGE = A_BYTES + B_BYTES;
  static constexpr int PATCH_OFF = STAGES * STAGE;
  static constexpr int BAR_OFF = PATCH_OFF + 4 * GB_PATCH;
  static constexpr int TOTAL = BAR_OFF + 256 + 1024;
};

template <int BN>
__global__ void __launch_bounds__(GB_THREADS, 1)
gemm_bf16_kernel(const __grid_constant__ CUtensorMap map_a, const __grid_constant__ CUtensorMap map_w, Bf16Product p, int m,
                 int m_tiles, int n_tiles, DevErr *err) {
  using L = GbSmem<BN>;
  constexpr int S = L::STAGES;
  extern __shared__ unsigned char smem_raw[];
  const unsigned base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  unsigned char *base_ptr = smem_raw + (base - smem_u32(smem_raw));
  const unsigned bars = base + L::BAR_OFF;
  auto full = [&](int s) { return bars + 8u * s; };
  auto empty = [&](int s) { return bars + 8u * (S + s); };
  auto tfull = [&](int b) { return bars + 8u * (2 * S + b); };
  auto tempty = [&](int b) { return bars + 8u * (2 * S + 2 + b); };
  volatile unsigned *tmem_holder = reinterpret_cast<volatile unsigned *>(base_ptr + L::BAR_OFF + 192);
  volatile int *abort_flag = reinterpret_cast<volatile int *>(base_ptr + L::BAR_OFF + 196);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tiles = m_tiles * n_tiles, kblocks = (p.k + 63) / 64;
  auto place = [&](int tile, int &m0, int &n0) {
    const int per = GB_GROUP * n_tiles, grp = tile / per, rest = tile - grp * per;
    const int gm = min(GB_GROUP, m_tiles - grp * GB_GROUP);
    n0 = rest / gm * BN;
    m0 = (grp * GB_GROUP + rest % gm) * TC_BM;
  };

  if (threadIdx.x == 0) {
    for (int s = 0; s < S; ++s) {
      mbar_init(full(s), 1);
      mbar_init(empty(s), 1);
    }
    for (int b = 0; b < 2; ++b) {
      mbar_init(tfull(b), 1);
      mbar_init(tempty(b), 4);
    }
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32((const void *)tmem_holder)),
                 "r"((unsigned)(2 * BN))
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const unsigned tmem = *tmem_holder;
  pdl_launch_dependents();  // behind the allocation: a dependent's CTA must not take tensor memory first
  pdl_wait();

  if (warp == 0) {
    int it = 0;
    bool ok = true;
    for (int tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x) {
      int m0, n0;
      place(tile, m0, n0);
      for (int kb = 0; kb < kblocks; ++kb, ++it) {
        const int s = it % S;
        ok = mbar_wait(empty(s), ((unsigned)(it / S) & 1u) ^ 1u, abort_flag, err, 11);
        __syncwarp();
        if (!ok) break;
        if (lane == 0) {
          const unsigned st = base + (unsigned)(s * L::STAGE);
          mbar_expect_tx(full(s), (unsigned)L::STAGE);
          tma_load_2d(st, &map_a, kb * 64, m0, full(s));
          tma_load_2d(st + L::A_BYTES, &map_w, kb * 64, n0, full(s));
        }
        __syncwarp();
      }
    }
    if (*abort_flag) {  // copies in flight must land before the shared memory goes away
      for (int j = it > S ? it - S : 0; j < it; ++j) {
        const unsigned long long t0 = global_timer();
        while (!mbar_try_wait(full(j % S), (unsigned)(j / S) & 1u))
          if (global_timer() - t0 > WAIT_LIMIT_NS) break;
      }
    }
  } else if (warp == 1) {
    constexpr unsigned idesc = umma_idesc_bf16(BN);
    int it = 0, use = 0;
    bool ok = true;
    for (int tile = blockIdx.x; tile < tiles && ok; tile += gridDim.x, ++use) {
      const int buf = use & 1;
      ok = mbar_wait(tempty(buf), ((unsigned)(use >> 1) & 1u) ^ 1u, abort_flag, err, 12);
      __syncwarp();
      if (!ok) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      for (int kb = 0; kb < kblocks; ++kb, ++it) {
        const int s = it % S;
        ok = mbar_wait(full(s), (unsigned)(it / S) & 1u, abort_flag, err, 13);
        __syncwarp();
        if (!ok) break;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        if (lane == 0) {
          const unsigned st = base + (unsigned)(s * L::STAGE);
          const unsigned long long da = umma_desc_k128(st), db = umma_desc_k128(st + L::A_BYTES);
#pragma unroll
          for (int ks = 0; ks < 4; ++ks)
            tc_mma_f16(tmem + (unsigned)(buf * BN), da + (unsigned long long)(ks * 2), db + (unsigned long long)(ks * 2), idesc,
                       (kb | ks) ? 1u : 0u);
          tc_commit(empty(s));
        }
        __syncwarp();
      }
      if (ok && lane == 0) tc_commit(tfull(buf));
      __syncwarp();
    }
    if (!ok) {  // give the tensor pipe a bounded chance to finish before tensor memory is freed
      const unsigned long long t0 = global_timer();
      if (lane == 0) tc_commit(tfull(use & 1));
      __syncwarp();
      while (!mbar_try_wait(tfull(use & 1), (unsigned)(use >> 1) & 1u))
        if (global_timer() - t0 > WAIT_LIMIT_NS) break;
    }
  } else {
    const int q = warp & 3;
    float *patch = reinterpret_cast<float *>(base_ptr + L::PATCH_OFF + (warp - 2) * GB_PATCH);
    const bool half_vec = p.half_out != nullptr && (p.half_ld & 3) == 0 && (reinterpret_cast<uintptr_t>(p.half_out) & 7) == 0;
    const bool float_vec = p.float_out != nullptr && (p.float_ld & 3) == 0 &&
                           (reinterpret_cast<uintptr_t>(p.float_out) & 15) == 0 && (p.n_half & 3) == 0;
    const int sub = lane >> 3, c4 = (lane & 7) * 4;
    int use = 0;
    for (int tile = blockIdx.x; tile < tiles; tile += gridDim.x, ++use) {
      const int buf = use & 1;
      if (!mbar_wait_warp(tfull(buf), (unsigned)(use >> 1) & 1u, abort_flag, err, 14)) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      int m0, n0;
      place(tile, m0, n0);
      const int row0 = m0 + q * 32;
#pragma unroll 1
      for (int c0 = 0; c0 < BN; c0 += 32) {
        unsigned r[32];
        tc_ld32(tmem + ((unsigned)(q * 32) << 16) + (unsigned)(buf * BN + c0), r);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
        if (c0 + 32 == BN) {
          asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
          __syncwarp();
          if (lane == 0) mbar_arrive(tempty(buf));
        }
        if (n0 + c0 >= p.n) continue;
        __syncwarp();
#pragma unroll
        for (int j = 0; j < 32; j += 4)
          *reinterpret_cast<uint4 *>(patch + lane * GB_PATCH_LD + j) = make_uint4(r[j], r[j + 1], r[j + 2], r[j + 3]);
        __syncwarp();
        const int col = n0 + c0 + c4;
        const bool to_half = col < p.n_half;
        const bool whole = col + 4 <= (to_half ? p.n_half : p.n);
#pragma unroll
        for (int i = 0; i < 8; ++i) {
          const int rr = i * 4 + sub, row = row0 + rr;
          if (row >= m || col >= p.n) continue;
          float4 v = *reinterpret_cast<const float4 *>(patch + rr * GB_PATCH_LD + c4);
          if (whole && to_half && p.gated) {  // two pairs
            const __nv_bfloat162 a = __floats2bfloat162_rn(activate(v.x, p.act) * v.y, activate(v.z, p.act) * v.w);
            *reinterpret_cast<__nv_bfloat162 *>(static_cast<bf16 *>(p.half_out) + (long long)row * p.half_ld + (col >> 1)) = a;
          } else if (whole && to_half && half_vec) {
            if (p.act != ACT_NONE)
              v = make_float4(activate(v.x, p.act), activate(v.y, p.act), activate(v.z, p.act), activate(v.w, p.act));
            const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
            uint2 o;
            o.x = *reinterpret_cast<const unsigned *>(&a);
            o.y = *reinterpret_cast<const unsigned *>(&b);
            *reinterpret_cast<uint2 *>(static_cast<bf16 *>(p.half_out) + (long long)row * p.half_ld + col) = o;
          } else if (whole && !to_half && float_vec) {
            float4 *o = reinterpret_cast<float4 *>(p.float_out + (long long)row * p.float_ld + (col - p.n_half));
            if (p.accumulate) {
              const float4 x = *o;
              v = make_float4(x.x + v.x, x.y + v.y, x.z + v.z, x.w + v.w);
            }
            *o = v;
          } else {
            const float e[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
            for (int j = 0; j < 4; ++j) {
              if (col + j >= p.n) continue;
              if (col + j < p.n_half) {
                if (p.gated) {
                  if ((j & 1) == 0)  // n_half is even
                    static_cast<bf16 *>(p.half_out)[(long long)row * p.half_ld + ((col + j) >> 1)] =
                        __float2bfloat16_rn(activate(e[j], p.act) * e[j + 1]);
                } else {
                  static_cast<bf16 *>(p.half_out)[(long long)row * p.half_ld + col + j] =
                      __float2bfloat16_rn(activate(e[j], p.act));
                }
              } else {
                float *o = p.float_out + (long long)row * p.float_ld + (col + j - p.n_half);
                *o = p.accumulate ? *o + e[j] : e[j];
              }
            }
          }
        }
      }
    }
  }
  __syncwarp();
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == 1) {
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"((unsigned)(2 * BN)));
  }
}

int device_sms() {
  static int n = 0;
  static std::once_flag once;
  std::call_once(once, [] {
    int dev = 0;
    cudaGetDevice(&dev);
    if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n <= 0) n = 148;
  });
  return n;
}

template <int BN>
void launch_bn(const Bf16Product &p, int m, cudaStream_t st, DevErr *err) {
  using L = GbSmem<BN>;
  CUtensorMap ma, mw;
  tc_make_map_bf16(&ma, p.a, (unsigned long long)m, (unsigned long long)p.k, (unsigned long long)p.a_ld, TC_BM);
  tc_make_map_bf16(&mw, p.w, (unsigned long long)p.n, (unsigned long long)p.k, (unsigned long long)p.w_ld, BN);
  LB_CUDA(cudaFuncSetAttribute(gemm_bf16_kernel<BN>, cudaFuncAttributeMaxDynamicSharedMemorySize, L::TOTAL));
  const int mt = (m + TC_BM - 1) / TC_BM, nt = (p.n + BN - 1) / BN;
  const long long tiles = (long long)mt * nt;
  const unsigned grid = (unsigned)(tiles < device_sms() ? tiles : device_sms());
  launch_pdl(gemm_bf16_kernel<BN>, dim3(grid), dim3(GB_THREADS), L::TOTAL, st, false, ma, mw, p, m, mt, nt, err);
}

}  // namespace

void launch_gemm_bf16(const Bf16Product &p, int m, cudaStream_t st, DevErr *err) {
  if (m < 1 || p.n < 1 || p.k < 1) throw std::invalid_argument("launch_gemm_bf16: empty product");
  if (p.gated && ((p.n_half | p.half_ld) & 1) != 0) throw std::invalid_argument("launch_gemm_bf16: a gated product needs pairs");
  // the widest tile that still gives most SMs one
  const long long mt = (m + TC_BM - 1) / TC_BM;
  const long long sms = device_sms();
  if (p.n > 128 && mt * ((p.n + 255) / 256) >= sms * 3 / 4) launch_bn<256>(p, m, st, err);
  else if (p.n > 64 && mt * ((p.n + 127) / 128) >= sms * 3 / 4) launch_bn<128>(p, m, st, err);
  else launch_bn<64>(p, m, st, err);
}

}  // namespace lb
