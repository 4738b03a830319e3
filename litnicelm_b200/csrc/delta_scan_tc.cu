// The chunks of the gated delta rule in order (delta_chunk.cu has the equations and prepares the matrices) on the
// sm_100a tensor cores: tcgen05 with every left operand and accumulator in tensor memory.
//
// One CTA per stream, head and 128 value columns. Tensor memory holds everything transposed, a lane per value column:
// S^T as a 32-bit accumulator that stays for the whole sequence, and the left operands as two bfloat16 terms each,
// written by the thread that owns the lane. So the elementwise steps between the products need no other thread, and
// the right operands are the shared-memory tiles as TMA brings them (128-byte swizzle):
//   PK = S^T K'^T, PQ = S^T Q'^T        right operand: K' and Q' rows
//   U  = (V^T - PK diag(e^G r)) T^T     right operand: T = (I + L)^-1 diag(beta), blocks of 16 on or below the diagonal
//   S^T <- e^G_last S^T + (U diag(e^(G_last - G) r)) K'      right operand: K' again, its dimensions contiguous
//   O  = PQ diag(e^G r') + U A^T        right operand: A
//
//   warp 0        TMA: K', Q', V tiles, the chunk's matrices and factors, two stages
//   warp 1        owns tensor memory and issues the products
//   warps 2-9     the chain: S to operand and decayed, right-hand side, U to operands; two warps share 32 lanes and take
//                 alternating blocks of 16 columns
//   warps 10-13   outputs, behind the chain: PQ scaled, O to shared memory, norm and gate over whole rows, store
// Every mbarrier wait is bounded; a wait that runs out sets the error word and ends the kernel after its copies have
// landed and tensor memory is freed. No clusters, no multicast.
#include "delta.cuh"
#include "gemm_tc.cuh"
#include "tc_ptx.cuh"

namespace lb {

namespace {

typedef __nv_bfloat16 bf16;

constexpr int CH = DELTA_CHUNK;
constexpr int DS_THREADS = 14 * 32;
constexpr int DS_CHAIN = 8, DS_OUT = 4;  // warps
constexpr int DS_BOX = CH * 128;         // 64 rows of 64 elements
constexpr int DS_SP = 132;               // floats per row of the output staging
// tensor-memory columns
constexpr unsigned TM_S = 0, TM_X = 128, TM_PK = 256, TM_PQ = 320, TM_U = 448;

struct DsArgs {
  DeltaChunks c;
  int p0, slot0, normed, in_ld, out_ld;
  float *state, *o;
  const bf16 *gate;
  float count, eps;
  const float *norm;
  bf16 *out;
};

// Byte offsets inside a stage.
struct DsStage {
  static constexpr int KQ = 0;                      // two slabs of [K' rows | Q' rows]
  static constexpr int V = KQ + 4 * DS_BOX;         // two slabs
  static constexpr int MATS = V + 2 * DS_BOX;       // T high, T low, A high, A low
  static constexpr int FACTORS = MATS + 4 * DS_BOX; // 64 float4
  static constexpr int BYTES = FACTORS + CH * 16;
};
constexpr int DS_STAGES_OFF = 0, DS_OUT_OFF = 2 * DsStage::BYTES, DS_BAR_OFF = DS_OUT_OFF + CH * DS_SP * 4;
constexpr int DS_SMEM = DS_BAR_OFF + 256 + 1024;

__device__ __forceinline__ unsigned pack2(float a, float b) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const unsigned *>(&v);
}
__device__ __forceinline__ float lowf(unsigned u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float highf(unsigned u) { return __uint_as_float(u & 0xffff0000u); }
// 16 floats as an operand block: eight columns of high terms, eight of low ones.
template <int AT>
__device__ __forceinline__ void operand_block(const float (&f)[16], unsigned *out) {
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    const unsigned hi = pack2(f[2 * i], f[2 * i + 1]);
    out[AT + i] = hi;
    out[AT + 8 + i] = pack2(f[2 * i] - lowf(hi), f[2 * i + 1] - highf(hi));
  }
}

__global__ void __launch_bounds__(DS_THREADS, 1)
delta_scan_tc_kernel(const __grid_constant__ CUtensorMap map_rows, const __grid_constant__ CUtensorMap map_mats, DsArgs s,
                     DevErr *err) {
  extern __shared__ unsigned char smem_raw[];
  const unsigned base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  unsigned char *base_ptr = smem_raw + (base - smem_u32(smem_raw));
  const DeltaChunks &a = s.c;
  const unsigned bars = base + DS_BAR_OFF;
  auto full = [&](int i) { return bars + 8u * i; };
  auto empty = [&](int i) { return bars + 8u * (2 + i); };
  auto pq_free = [&](int i) { return bars + 8u * (4 + i); };
  const unsigned sh_ready = bars + 48, pk_full = bars + 56, pq_full = bars + 64, r_ready = bars + 72, u_full = bars + 80,
                 uh_ready = bars + 88, s_full = bars + 96, pq_scaled = bars + 104, o_full = bars + 112, rows_in = bars + 120,
                 rows_out = bars + 128;
  volatile unsigned *tmem_holder = reinterpret_cast<volatile unsigned *>(base_ptr + DS_BAR_OFF + 192);
  volatile int *abort_flag = reinterpret_cast<volatile int *>(base_ptr + DS_BAR_OFF + 196);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tiles = (a.vdim + 127) / 128;
  const int h = blockIdx.x / tiles, vt = (blockIdx.x - h * tiles) * 128, b = blockIdx.y;
  const int grp = h / (a.heads / a.groups), vcols = min(128, a.vdim - vt);
  const int slabs = (a.dim + 63) >> 6, vslabs = (vcols + 63) >> 6, blocks = a.dim >> 4;
  auto stage_ptr = [&](int c) { return base_ptr + DS_STAGES_OFF + (c & 1) * DsStage::BYTES; };
  auto factors_of = [&](int c) { return reinterpret_cast<const float4 *>(stage_ptr(c) + DsStage::FACTORS); };

  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; ++i) {
      mbar_init(full(i), 1);
      mbar_init(empty(i), 1 + DS_CHAIN + DS_OUT);
      mbar_init(pq_free(i), DS_OUT);
    }
    for (unsigned bar : {pk_full, pq_full, u_full, s_full, o_full}) mbar_init(bar, 1);
    for (unsigned bar : {sh_ready, r_ready, uh_ready}) mbar_init(bar, DS_CHAIN);
    for (unsigned bar : {pq_scaled, rows_in, rows_out}) mbar_init(bar, DS_OUT);
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32((const void *)tmem_holder)),
                 "r"(512u)
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
    bool ok = true;
    int loads = 0;
    for (int c = 0; c < a.chunks && ok; ++c) {
      const int i = c & 1;
      ok = mbar_wait_warp(empty(i), ((unsigned)(c >> 1) & 1u) ^ 1u, abort_flag, err, 41);
      if (!ok) break;
      if (lane == 0) {
        const unsigned st = base + DS_STAGES_OFF + (unsigned)(i * DsStage::BYTES);
        const int row = b * a.n + c * CH, at = (b * a.heads + h) * a.chunks + c;
        mbar_expect_tx(full(i), (unsigned)((2 * slabs + vslabs + 4) * DS_BOX + CH * 16));
        for (int k = 0; k < slabs; ++k) {
          tma_load_2d(st + DsStage::KQ + k * 2 * DS_BOX, &map_rows, (a.groups + grp) * a.dim + k * 64, row, full(i));
          tma_load_2d(st + DsStage::KQ + (k * 2 + 1) * DS_BOX, &map_rows, grp * a.dim + k * 64, row, full(i));
        }
        for (int k = 0; k < vslabs; ++k)
          tma_load_2d(st + DsStage::V + k * DS_BOX, &map_rows, 2 * a.groups * a.dim + h * a.vdim + vt + k * 64, row, full(i));
        for (int k = 0; k < 4; ++k) tma_load_2d(st + DsStage::MATS + k * DS_BOX, &map_mats, 0, (at * 4 + k) * CH, full(i));
        bulk_load(st + DsStage::FACTORS, a.factors + (long long)at * CH, CH * 16, full(i));
      }
      ++loads;
      __syncwarp();
    }
    if (*abort_flag) {  // copies in flight must land before the shared memory goes away
      const unsigned long long limit = global_timer() + WAIT_LIMIT_NS;
      for (int c = loads > 2 ? loads - 2 : 0; c < loads; ++c)
        while (!mbar_try_wait(full(c & 1), (unsigned)(c >> 1) & 1u) && global_timer() < limit) {}
    }
  } else if (warp == 1) {
    const unsigned id64 = umma_idesc_bf16(CH), id_s = umma_idesc_bf16(a.dim) | UMMA_B_MN_MAJOR;
    bool ok = true;
    int c = 0;
    auto hold = [&](unsigned bar, unsigned parity, int where) {
      ok = ok && mbar_wait_warp(bar, parity, abort_flag, err, where);
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      return ok;
    };
    // D[:, 16 kt ..] += A blocks (high at x, low at x + 8) times a lower triangular matrix's rows 16 kt .. of both terms
    auto triangle = [&](unsigned d, unsigned x, unsigned step, unsigned mat, bool fresh) {
#pragma unroll
      for (int kt = 0; kt < 4; ++kt) {
        const unsigned long long hi = umma_desc_k128(mat + (unsigned)(kt * 2048)) + (unsigned long long)(kt * 2);
        const unsigned long long lo = umma_desc_k128(mat + DS_BOX + (unsigned)(kt * 2048)) + (unsigned long long)(kt * 2);
        const unsigned id = umma_idesc_bf16(CH - 16 * kt), at = d + (unsigned)(16 * kt), op = x + (unsigned)kt * step;
        tc_mma_f16_ts(at, op, hi, id, fresh && kt == 0 ? 0u : 1u);
        tc_mma_f16_ts(at, op, lo, id, 1u);
        tc_mma_f16_ts(at, op + 8, hi, id, 1u);
      }
    };
    for (; c < a.chunks; ++c) {
      const unsigned st = base + DS_STAGES_OFF + (unsigned)((c & 1) * DsStage::BYTES), ph = (unsigned)c & 1u;
      if (!hold(full(c & 1), (unsigned)(c >> 1) & 1u, 42) || !hold(sh_ready, ph, 43)) break;
      auto state_product = [&](unsigned d, unsigned rows) {
        for (int ks = 0; ks < blocks; ++ks) {
          const unsigned long long x = umma_desc_k128(rows + (unsigned)((ks >> 2) * 2 * DS_BOX)) + (unsigned long long)((ks & 3) * 2);
          tc_mma_f16_ts(d, tmem + TM_X + (unsigned)(ks * 16), x, id64, ks ? 1u : 0u);
          tc_mma_f16_ts(d, tmem + TM_X + (unsigned)(ks * 16 + 8), x, id64, 1u);
        }
      };
      if (lane == 0) {
        state_product(tmem + TM_PK, st + DsStage::KQ);
        tc_commit(pk_full);
      }
      __syncwarp();
      if (c >= 2 && !hold(pq_free(c & 1), (unsigned)((c >> 1) - 1) & 1u, 44)) break;
      const unsigned pq = tmem + TM_PQ + (unsigned)((c & 1) * CH);
      if (lane == 0) {
        state_product(pq, st + DsStage::KQ + DS_BOX);
        tc_commit(pq_full);
      }
      __syncwarp();
      if (!hold(r_ready, ph, 45)) break;
      if (lane == 0) {
        triangle(tmem + TM_U, tmem + TM_PK, 16, st + DsStage::MATS, true);
        tc_commit(u_full);
      }
      __syncwarp();
      if (!hold(uh_ready, ph, 46)) break;
      if (lane == 0) {
#pragma unroll
        for (int kt = 0; kt < 4; ++kt) {
          const unsigned long long x = umma_desc_mn128(st + DsStage::KQ + (unsigned)(kt * 2048), 2 * DS_BOX);
          tc_mma_f16_ts(tmem + TM_S, tmem + TM_X + (unsigned)(kt * 32 + 16), x, id_s, 1u);
          tc_mma_f16_ts(tmem + TM_S, tmem + TM_X + (unsigned)(kt * 32 + 24), x, id_s, 1u);
        }
        tc_commit(s_full);
      }
      __syncwarp();
      if (!hold(pq_scaled, ph, 47)) break;
      if (lane == 0) {
        triangle(pq, tmem + TM_X, 32, st + DsStage::MATS + 2 * DS_BOX, false);
        tc_commit(o_full);
        tc_commit(empty(c & 1));
      }
      __syncwarp();
    }
    if (!ok) {  // a bounded chance for the tensor pipe to finish before tensor memory is freed
      if (lane == 0) tc_commit(o_full);
      __syncwarp();
      const unsigned long long limit = global_timer() + WAIT_LIMIT_NS;
      while (!mbar_try_wait(o_full, (unsigned)c & 1u) && global_timer() < limit) {}
    }
  } else if (warp < 2 + DS_CHAIN) {
    const int q = warp & 3, half = (warp - 2) >> 2;
    const unsigned lanes = tmem + ((unsigned)(q * 32) << 16);
    const int vl = q * 32 + lane, v = vt + vl;  // this thread's value column
    const bool mine = vl < vcols;
    float *S = s.state + ((long long)(s.slot0 + b) * a.heads + h) * a.dim * a.vdim + v;
    bool ok = true;
    auto hold = [&](unsigned bar, unsigned parity, int where) {
      ok = ok && mbar_wait_warp(bar, parity, abort_flag, err, where);
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      return ok;
    };
    auto release = [&](unsigned bar) {
      asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      __syncwarp();
      if (lane == 0) mbar_arrive(bar);
    };
    for (int c = 0; c < a.chunks && ok; ++c) {
      const unsigned ph = (unsigned)c & 1u;
      // S: operand blocks for the products with K' and Q', and e^G_last S in place
      unsigned x[4][16];
      if (c == 0) {
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 16; ++j) {
            const int d = (2 * i + half) * 16 + j;
            x[i][j] = s.p0 > 0 && mine && d < a.dim ? __float_as_uint(S[(long long)d * a.vdim]) : 0u;
          }
      } else {
        if (!hold(s_full, ph ^ 1u, 48)) break;
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (2 * i + half < blocks) tc_ld16(lanes + TM_S + (unsigned)((2 * i + half) * 16), x[i]);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
      }
      if (!hold(full(c & 1), (unsigned)(c >> 1) & 1u, 49)) break;
      const float4 *fs = factors_of(c);
      const float keep = fs[0].w;
      if (c > 0 && !hold(o_full, ph ^ 1u, 50)) break;  // U's operands are read: their columns are S's now
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int kt = 2 * i + half;
        if (kt < blocks) {
          float f[16];
          unsigned w[16];
#pragma unroll
          for (int j = 0; j < 16; ++j) f[j] = __uint_as_float(x[i][j]);
          operand_block<0>(f, w);
          tc_st16(lanes + TM_X + (unsigned)(kt * 16), w);
#pragma unroll
          for (int j = 0; j < 16; ++j) w[j] = __float_as_uint(f[j] * keep);
          tc_st16(lanes + TM_S + (unsigned)(kt * 16), w);
        }
      }
      release(sh_ready);
      // right-hand side, over the columns it is made of
      const unsigned char *vs = stage_ptr(c) + DsStage::V + (vl >> 6) * DS_BOX;
      float rhs[2][16];
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 16; ++j) {
          const int t = (2 * i + half) * 16 + j;
          rhs[i][j] = mine ? __bfloat162float(*reinterpret_cast<const bf16 *>(vs + t * 128 + (((vl & 63) * 2) ^ ((t & 7) << 4)))) : 0.f;
        }
      if (!hold(pk_full, ph, 51)) break;
#pragma unroll
      for (int i = 0; i < 2; ++i) tc_ld16(lanes + TM_PK + (unsigned)((2 * i + half) * 16), x[i]);
      asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int kt = 2 * i + half;
        unsigned w[16];
#pragma unroll
        for (int j = 0; j < 16; ++j) rhs[i][j] = fmaf(-fs[kt * 16 + j].x, __uint_as_float(x[i][j]), rhs[i][j]);
        operand_block<0>(rhs[i], w);
        tc_st16(lanes + TM_PK + (unsigned)(kt * 16), w);
      }
      release(r_ready);
      // U as it is (for the outputs) and brought to the chunk's end (for the state)
      if (!hold(u_full, ph, 52)) break;
#pragma unroll
      for (int i = 0; i < 2; ++i) tc_ld16(lanes + TM_U + (unsigned)((2 * i + half) * 16), x[i]);
      asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int kt = 2 * i + half;
        float f[16];
        unsigned w[32];
#pragma unroll
        for (int j = 0; j < 16; ++j) f[j] = __uint_as_float(x[i][j]);
        operand_block<0>(f, w);
#pragma unroll
        for (int j = 0; j < 16; ++j) f[j] *= fs[kt * 16 + j].z;
        operand_block<16>(f, w);
        tc_st32(lanes + TM_X + (unsigned)(kt * 32), w);
      }
      release(uh_ready);
      if (lane == 0) mbar_arrive(empty(c & 1));
    }
    if (ok && hold(s_full, (unsigned)(a.chunks - 1) & 1u, 53)) {
      unsigned x[4][16];
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (2 * i + half < blocks) tc_ld16(lanes + TM_S + (unsigned)((2 * i + half) * 16), x[i]);
      asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 16; ++j) {
          const int d = (2 * i + half) * 16 + j;
          if (mine && d < a.dim) S[(long long)d * a.vdim] = __uint_as_float(x[i][j]);
        }
    }
  } else {
    const int q = warp & 3, tid = threadIdx.x - (2 + DS_CHAIN) * 32;
    const unsigned lanes = tmem + ((unsigned)(q * 32) << 16);
    const int vl = q * 32 + lane;
    float *staging = reinterpret_cast<float *>(base_ptr + DS_OUT_OFF);
    bool ok = true;
    auto hold = [&](unsigned bar, unsigned parity, int where) {
      ok = ok && mbar_wait_warp(bar, parity, abort_flag, err, where);
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      return ok;
    };
    auto release = [&](unsigned bar) {
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      __syncwarp();
      if (lane == 0) mbar_arrive(bar);
    };
    // whole rows of outputs: 16 lanes per token, eight columns each, eight tokens at a time
    const int col = (tid & 15) * 8, row0 = tid >> 4;
    const bool in = col < vcols;
    float4 w0 = make_float4(0.f, 0.f, 0.f, 0.f), w1 = w0;
    if (s.normed && in) {
      w0 = *reinterpret_cast<const float4 *>(s.norm + col);
      w1 = *reinterpret_cast<const float4 *>(s.norm + col + 4);
    }
    for (int c = 0; c < a.chunks && ok; ++c) {
      const unsigned ph = (unsigned)c & 1u, pq = lanes + TM_PQ + (unsigned)((c & 1) * CH);
      const int t0 = c * CH, nt = min(CH, a.n - t0);
      uint4 gate[8];
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int t = row0 + 8 * k;
        gate[k] = s.normed && in && t < nt
                      ? *reinterpret_cast<const uint4 *>(s.gate + ((long long)b * a.n + t0 + t) * s.in_ld + h * a.vdim + col)
                      : make_uint4(0, 0, 0, 0);
      }
      if (!hold(full(c & 1), (unsigned)(c >> 1) & 1u, 54) || !hold(pq_full, ph, 55)) break;
      const float4 *fs = factors_of(c);
      unsigned x[2][32];
#pragma unroll
      for (int i = 0; i < 2; ++i) tc_ld32(pq + (unsigned)(i * 32), x[i]);
      asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
      for (int i = 0; i < 2; ++i) {
#pragma unroll
        for (int j = 0; j < 32; ++j) x[i][j] = __float_as_uint(__uint_as_float(x[i][j]) * fs[i * 32 + j].y);
        tc_st32(pq + (unsigned)(i * 32), x[i]);
      }
      asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      release(pq_scaled);
      if (lane == 0) mbar_arrive(empty(c & 1));
      if (!hold(o_full, ph, 56)) break;
#pragma unroll
      for (int i = 0; i < 2; ++i) tc_ld32(pq + (unsigned)(i * 32), x[i]);
      asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
      release(pq_free(c & 1));
      if (c > 0 && !hold(rows_out, ph ^ 1u, 57)) break;  // the last chunk's rows have been read
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 32; ++j) staging[(i * 32 + j) * DS_SP + vl] = vl < vcols ? __uint_as_float(x[i][j]) : 0.f;
      release(rows_in);
      if (!hold(rows_in, ph, 58)) break;
#pragma unroll
      for (int k = 0; k < 8; ++k) {
        const int t = row0 + 8 * k;
        const float4 y = *reinterpret_cast<const float4 *>(staging + t * DS_SP + col);
        const float4 z = *reinterpret_cast<const float4 *>(staging + t * DS_SP + col + 4);
        const long long r = (long long)b * a.n + t0 + t;
        if (!s.normed) {
          if (in && t < nt) {
            float *o = s.o + (r * a.heads + h) * a.vdim + vt + col;
            *reinterpret_cast<float4 *>(o) = y;
            *reinterpret_cast<float4 *>(o + 4) = z;
          }
          continue;
        }
        float sum = y.x * y.x + y.y * y.y + y.z * y.z + y.w * y.w + z.x * z.x + z.y * z.y + z.z * z.z + z.w * z.w;
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        if (!in || t >= nt) continue;
        const float inv = 1.0f / sqrtf(sum / s.count + s.eps);
        const uint4 g = gate[k];
        *reinterpret_cast<uint4 *>(s.out + r * s.out_ld + h * a.vdim + col) =
            make_uint4(pack2(y.x * inv * w0.x * silu_fast(lowf(g.x)), y.y * inv * w0.y * silu_fast(highf(g.x))),
                       pack2(y.z * inv * w0.z * silu_fast(lowf(g.y)), y.w * inv * w0.w * silu_fast(highf(g.y))),
                       pack2(z.x * inv * w1.x * silu_fast(lowf(g.z)), z.y * inv * w1.y * silu_fast(highf(g.z))),
                       pack2(z.z * inv * w1.z * silu_fast(lowf(g.w)), z.w * inv * w1.w * silu_fast(highf(g.w))));
      }
      release(rows_out);
    }
  }
  __syncwarp();
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == 1) {
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(512u));
  }
}

}  // namespace

bool delta_scan_tc_supports(const DeltaMixer &m) { return m.dim <= 128 && m.vdim > 64; }

bool launch_delta_scan_tc(const DeltaMixer &m, const DeltaChunks &c, float *o, const RowBatch &b, cudaStream_t st, DevErr *err) {
  DsArgs s{};
  s.c = c;
  s.p0 = b.p0;
  s.slot0 = b.slot0;
  s.normed = m.vdim <= 128;
  s.in_ld = m.in_ld;
  s.out_ld = m.out_ld;
  s.state = m.state;
  s.o = o;
  s.gate = static_cast<const bf16 *>(m.in) + c.channels;
  s.count = (float)m.true_vdim;
  s.eps = m.eps;
  s.norm = m.norm;
  s.out = static_cast<bf16 *>(m.out);
  CUtensorMap rows, mats;
  tc_make_map_bf16(&rows, c.conv, (unsigned long long)b.rows(), (unsigned long long)c.channels, (unsigned long long)c.channels, CH);
  tc_make_map_bf16(&mats, c.mats, (unsigned long long)b.streams * c.heads * c.chunks * 4 * CH, CH, CH, CH);
  LB_CUDA(cudaFuncSetAttribute(delta_scan_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, DS_SMEM));
  launch_pdl(delta_scan_tc_kernel, dim3((unsigned)(m.heads * ((m.vdim + 127) / 128)), (unsigned)b.streams), dim3(DS_THREADS),
             (size_t)DS_SMEM, st, g_pdl_enabled, rows, mats, s, err);
  return s.normed != 0;
}

}  // namespace lb
