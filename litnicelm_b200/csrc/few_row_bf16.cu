// Few-row products on bfloat16 weights: C[m, n] = A[m, k] W[n, k]^T for m <= 64 rows, bound by the
// bytes of W, which every launch reads once.
//
// W rows are the M side of mma.sync m16n8k16 tiles and the activation rows the N side, so one
// instruction serves 16 output columns and 8 rows. A CTA owns 16 rows of W and all of k; its eight
// warps take interleaved blocks of 64 k, and their sums meet in shared memory. The order of k inside a
// dot product is free, so a lane loads 16 consecutive bytes (8 k) of its W row and of its activation
// row and feeds them to two k-steps as they lie: no shared memory, no shuffles, whole 128-byte lines
// of W per warp and row. Up to two products with inputs of their own share a launch. Where the columns
// alone give too few CTAs, k is cut over the CTAs of a thread-block cluster, whose sums meet in the shared
// memory of the rank that stores them (rank order, so results do not depend on scheduling).
#include "activation.cuh"
#include "model.cuh"
#include "tc_ptx.cuh"

#include <cuda_bf16.h>

namespace lb {

namespace {

typedef __nv_bfloat16 bf16;

constexpr int FR_WARPS = 8;
constexpr int FR_COLS = 16;  // rows of W (output columns) per CTA

struct FewRowPair {
  Bf16Product p[2];
  int blocks0;  // CTAs of the first product
};

__device__ __forceinline__ void fr_mma(float (&d)[4], unsigned a0, unsigned a1, unsigned a2, unsigned a3, unsigned b0,
                                       unsigned b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint4 ld_stream(const bf16 *p) {  // weights: read once per launch
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];"
               : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w)
               : "l"(p));
  return v;
}

// NT: tiles of 8 activation rows; UNROLL: blocks of 32 k in flight per lane and row.
template <int NT, int UNROLL>
__global__ void __launch_bounds__(FR_WARPS * 32)
few_row_bf16_kernel(FewRowPair pair, int m, int ranks) {
  __shared__ __align__(16) float red[FR_WARPS][NT][FR_COLS][8];
  const bool second = (int)blockIdx.x >= pair.blocks0;
  const Bf16Product &p = pair.p[second ? 1 : 0];
  const int n0 = ((int)blockIdx.x - (second ? pair.blocks0 : 0)) * FR_COLS;
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
  const int k8 = (p.k + 7) & ~7;  // rows end on a multiple of 8, zeros behind k
  const bf16 *w = static_cast<const bf16 *>(p.w), *a = static_cast<const bf16 *>(p.a);
  const bool v0 = n0 + g < p.n, v1 = n0 + g + 8 < p.n;
  const bf16 *w0 = w + (long long)(n0 + g) * p.w_ld + t * 8, *w1 = w0 + (long long)8 * p.w_ld;
  constexpr int SPAN = 32 * UNROLL;  // k per warp and trip
  // this CTA's range of k, in whole spans
  const int per = ((k8 + SPAN - 1) / SPAN + ranks - 1) / ranks * SPAN;
  const int k_begin = min(k8, (int)blockIdx.z * per), k_end = min(k8, k_begin + per);
  const uint4 zero = make_uint4(0, 0, 0, 0);
  uint4 wa[UNROLL], wb[UNROLL];
  auto load_w = [&](int k0) {
#pragma unroll
    for (int u = 0; u < UNROLL; ++u) {
      const int k = k0 + u * 32;
      const bool in = k + t * 8 < k_end;
      wa[u] = in && v0 ? ld_stream(w0 + k) : zero;
      wb[u] = in && v1 ? ld_stream(w1 + k) : zero;
    }
  };
  float acc[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
  pdl_launch_dependents();
  load_w(k_begin + wid * SPAN);  // the weights do not depend on the predecessor
  pdl_wait();
  for (int k0 = k_begin + wid * SPAN; k0 < k_end; k0 += FR_WARPS * SPAN) {
    if constexpr (NT >= 8) {  // one tile's activations of all blocks at a time: fewer registers
#pragma unroll
      for (int i = 0; i < NT; ++i) {
        const int row = i * 8 + g;
        const bf16 *ar = a + (long long)row * p.a_ld + t * 8;
        uint4 x[UNROLL];
#pragma unroll
        for (int u = 0; u < UNROLL; ++u) {
          const int k = k0 + u * 32;
          x[u] = row < m && k + t * 8 < k_end ? *reinterpret_cast<const uint4 *>(ar + k) : zero;
        }
#pragma unroll
        for (int u = 0; u < UNROLL; ++u) {
          fr_mma(acc[i], wa[u].x, wb[u].x, wa[u].y, wb[u].y, x[u].x, x[u].y);
          fr_mma(acc[i], wa[u].z, wb[u].z, wa[u].w, wb[u].w, x[u].z, x[u].w);
        }
      }
    } else {
      // all tiles' activations of a block of 32 k are requested together, one block ahead of their use
      uint4 x[2][NT];
      auto load_x = [&](int u, uint4 (&dst)[NT]) {
        const int k = k0 + u * 32 + t * 8;
#pragma unroll
        for (int i = 0; i < NT; ++i)
          dst[i] = i * 8 + g < m && k < k_end ? *reinterpret_cast<const uint4 *>(a + (long long)(i * 8 + g) * p.a_ld + k) : zero;
      };
      load_x(0, x[0]);
#pragma unroll
      for (int u = 0; u < UNROLL; ++u) {
        if (u + 1 < UNROLL) load_x(u + 1, x[(u + 1) & 1]);
#pragma unroll
        for (int i = 0; i < NT; ++i) {
          const uint4 v = x[u & 1][i];
          fr_mma(acc[i], wa[u].x, wb[u].x, wa[u].y, wb[u].y, v.x, v.y);
          fr_mma(acc[i], wa[u].z, wb[u].z, wa[u].w, wb[u].w, v.z, v.w);
        }
      }
    }
    if (k0 + FR_WARPS * SPAN < k_end) load_w(k0 + FR_WARPS * SPAN);
  }
#pragma unroll
  for (int i = 0; i < NT; ++i) {
    *reinterpret_cast<float2 *>(&red[wid][i][g][t * 2]) = make_float2(acc[i][0], acc[i][1]);
    *reinterpret_cast<float2 *>(&red[wid][i][g + 8][t * 2]) = make_float2(acc[i][2], acc[i][3]);
  }
  __syncthreads();
  constexpr int TILE = NT * FR_COLS * 8;  // one warp's sums
  int e_begin = 0, e_end = TILE;
  if (ranks > 1) {  // the warps' sums first, in place; each rank then finishes its share of the tile
    float *flat = &red[0][0][0][0];
    for (int e = threadIdx.x; e < TILE; e += FR_WARPS * 32) {
      float v = 0.f;
#pragma unroll
      for (int q = 0; q < FR_WARPS; ++q) v += flat[q * TILE + e];
      flat[e] = v;  // this thread alone reads and writes element e of every warp
    }
    __syncwarp();
    cluster_sync_all();
    const int share = (TILE + ranks - 1) / ranks;
    e_begin = min(TILE, (int)blockIdx.z * share);
    e_end = min(TILE, e_begin + share);
  }
  auto total = [&](int c, int row) {
    float v = 0.f;
    if (ranks > 1) {
      const unsigned at = smem_u32(&red[0][row >> 3][c][row & 7]);
      for (int q = 0; q < ranks; ++q) v += ld_cluster_f32(cluster_map(at, (unsigned)q));
    } else {
#pragma unroll
      for (int q = 0; q < FR_WARPS; ++q) v += red[q][row >> 3][c][row & 7];
    }
    return v;
  };
  for (int e = e_begin + threadIdx.x; e < e_end; e += FR_WARPS * 32) {
    const int c = e & (FR_COLS - 1), row = e / FR_COLS;
    const int col = n0 + c;
    if (row >= m || col >= p.n) continue;
    if (p.gated && col < p.n_half) {  // a pair's columns are neighbours in one share: its even one finishes both
      if (c & 1) continue;
      const float z = activate(total(c, row), p.act) * total(c + 1, row);
      static_cast<bf16 *>(p.half_out)[(long long)row * p.half_ld + (col >> 1)] = __float2bfloat16_rn(z);
      continue;
    }
    const float v = total(c, row);
    if (col < p.n_half) {
      static_cast<bf16 *>(p.half_out)[(long long)row * p.half_ld + col] = __float2bfloat16_rn(activate(v, p.act));
    } else {
      float *o = p.float_out + (long long)row * p.float_ld + (col - p.n_half);
      *o = p.accumulate ? *o + v : v;
    }
  }
  __syncwarp();
  if (ranks > 1) cluster_sync_all();  // a rank's shared memory stays until every other has read it
}

}  // namespace

void launch_few_row_bf16(const Bf16Product *p, int count, int m, cudaStream_t st) {
  if (m < 1 || m > FEW_ROWS_MAX || count < 1 || count > 2) throw std::invalid_argument("launch_few_row_bf16: bad shape");
  FewRowPair pair{};
  unsigned blocks = 0;
  for (int i = 0; i < count; ++i) {
    pair.p[i] = p[i];
    blocks += (unsigned)((p[i].n + FR_COLS - 1) / FR_COLS);
    if (i == 0) pair.blocks0 = (int)blocks;
  }
  int k_max = 0;
  for (int i = 0; i < count; ++i) k_max = p[i].k > k_max ? p[i].k : k_max;
  // ranks of a cluster that share a tile's k: enough CTAs for two per SM, at least 512 k each
  int ranks = 1;
  const int ranks_max = m > 16 ? 4 : 8;  // many rows: a CTA's share of the sums is work too
  while (ranks < ranks_max && blocks * ranks < 2 * 148 && k_max >= 1024 * ranks) ranks *= 2;
  const dim3 grid(blocks, 1, (unsigned)ranks), block(FR_WARPS * 32);
  auto go = [&](auto kernel) {
    launch_pdl_cluster(kernel, grid, block, 0, st, g_pdl_enabled, (unsigned)ranks, pair, m, ranks);
  };
  const int nt = (m + 7) / 8;
  if (ranks > 1) {  // shorter ranges: two blocks of 32 k per lane and trip keep every warp busy
    if (nt <= 1) go(few_row_bf16_kernel<1, 2>);
    else if (nt <= 2) go(few_row_bf16_kernel<2, 2>);
    else if (nt <= 4) go(few_row_bf16_kernel<4, 2>);
    else go(few_row_bf16_kernel<8, 4>);
    return;
  }
  if (nt <= 1) go(few_row_bf16_kernel<1, 4>);
  else if (nt <= 2) go(few_row_bf16_kernel<2, 4>);
  else if (nt <= 4) go(few_row_bf16_kernel<4, 4>);
  else go(few_row_bf16_kernel<8, 4>);
}

}  // namespace lb
