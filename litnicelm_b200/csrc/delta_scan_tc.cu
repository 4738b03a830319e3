// The chunks of the gated delta rule in order (delta_chunk.cu has the equations and prepares the matrices) on the
// sm_100a tensor cores: tcgen05 with every left operand and accumulator in tensor memory.
//
// One CTA per stream, head and 128 value columns. Tensor memory holds everything transposed, a lane per value column:
// S^T as a 32-bit accumulator that stays for the whole sequence, and the left operands as two bfloat16 terms each,
// written by the thread that owns the lane. So the elementwise steps between the products need no other thread, and
// the right operands are the shared-memory tiles as TMA brings them (128-byte swizzle):
//   [PK | PQ] = S^T [K'^T | Q'^T]       right operand: K' and Q' rows
//   U  = (V^T - PK diag(e^G r)) T^T     right operand: T = (I + L)^-1 diag(beta), blocks of 16 on or below the diagonal
//   S^T <- e^G_last S^T + (U diag(e^(G_last - G) r)) K'      right operand: K' again, its dimensions contiguous
//   UA = U A^T                          right operand: A;  the output is PQ diag(e^G r') + UA
// Columns serve one thing after another: the operand of S becomes U, PK the right-hand side and then UA.
//
//   warp 0        TMA: K', Q', V tiles, the chunk's matrices and factors, two stages
//   warp 1        owns tensor memory and issues the products
//   warps 2-9     the chain: S to operand and decayed, right-hand side, U to operands; two warps share 32 lanes and take
//                 alternating blocks of 16 columns
//   warps 10-17   outputs, behind the chain: to shared memory, norm and gate over whole rows, store
// Every mbarrier wait is bounded; a wait that runs out sets the error word and ends the kernel after its copies have
// landed and tensor memory is freed. No clusters, no multicast.
#include "delta.cuh"
#include "gemm_tc.cuh"
#include "tc_ptx.cuh"

namespace lb {

namespace {

typedef __nv_bfloat16 bf16;

constexpr int CH = DELTA_CHUNK;
constexpr int DS_CHAIN = 8, DS_OUT = 8;  // warps
constexpr int DS_THREADS = (2 + DS_CHAIN + DS_OUT) * 32;
constexpr int DS_PIECES = CH * 16 / (DS_OUT * 32);  // pieces of eight outputs per thread
constexpr int DS_BOX = CH * 128;         // 64 rows of 64 elements
constexpr int DS_SP = 132;               // floats per row of the output staging
// tensor-memory columns
constexpr unsigned TM_S = 0, TM_SH = 128, TM_UH = 256, TM_PK = 384, TM_PQ = 448, TM_U = TM_SH, TM_UA = TM_PK;

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
  static constexpr int FACTORS = MATS + 4 * DS_BOX; // [4][64] floats
  static constexpr int BYTES = FACTORS + CH * 16;
};
constexpr int DS_STAGES_OFF = 0, DS_OUT_OFF = 2 * DsStage::BYTES, DS_GATE_OFF = DS_OUT_OFF + CH * DS_SP * 4,
              DS_BAR_OFF = DS_GATE_OFF + DS_PIECES * DS_OUT * 32 * 16;
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
  const unsigned sh_ready = bars + 32, p_full = bars + 40, r_ready = bars + 48, u_full = bars + 56, uh_ready = bars + 64,
                 s_full = bars + 72, o_full = bars + 80, o_read = bars + 88, rows_in = bars + 96, rows_out = bars + 104;
  volatile unsigned *tmem_holder = reinterpret_cast<volatile unsigned *>(base_ptr + DS_BAR_OFF + 192);
  volatile int *abort_flag = reinterpret_cast<volatile int *>(base_ptr + DS_BAR_OFF + 196);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int tiles = (a.vdim + 127) / 128;
  const int h = blockIdx.x / tiles, vt = (blockIdx.x - h * tiles) * 128, b = blockIdx.y;
  const int grp = h / (a.heads / a.groups), vcols = min(128, a.vdim - vt);
  const int slabs = (a.dim + 63) >> 6, vslabs = (vcols + 63) >> 6, blocks = a.dim >> 4;
  auto stage_ptr = [&](int c) { return base_ptr + DS_STAGES_OFF + (c & 1) * DsStage::BYTES; };
  auto factors_of = [&](int c) { return reinterpret_cast<const float *>(stage_ptr(c) + DsStage::FACTORS); };

  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; ++i) {
      mbar_init(full(i), 1);
      mbar_init(empty(i), 1 + DS_CHAIN + DS_OUT);
    }
    for (unsigned bar : {p_full, u_full, s_full, o_full}) mbar_init(bar, 1);
    for (unsigned bar : {sh_ready, r_ready, uh_ready}) mbar_init(bar, DS_CHAIN);
    for (unsigned bar : {o_read, rows_in, rows_out}) mbar_init(bar, DS_OUT);
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
        bulk_load(st + DsStage::FACTORS, a.factors + (long long)at * 4 * CH, CH * 16, full(i));
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
    const unsigned id_p = umma_idesc_bf16(2 * CH), id_s = umma_idesc_bf16(a.dim) | UMMA_B_MN_MAJOR;
    bool ok = true;
    int c = 0;
    auto hold = [&](unsigned bar, unsigned parity, int where) {
      ok = ok && mbar_wait_warp(bar, parity, abort_flag, err, where);
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      return ok;
    };
    // D[:, 16 kt ..] (+)= operand blocks (high at x, low at x + 8) times a lower triangular matrix's rows 16 kt .. of both
    // terms
    auto triangle = [&](unsigned d, unsigned x, unsigned step, unsigned mat) {
#pragma unroll
      for (int kt = 0; kt < 4; ++kt) {
        const unsigned long long hi = umma_desc_k128(mat + (unsigned)(kt * 2048)) + (unsigned long long)(kt * 2);
        const unsigned long long lo = umma_desc_k128(mat + DS_BOX + (unsigned)(kt * 2048)) + (unsigned long long)(kt * 2);
        const unsigned id = umma_idesc_bf16(CH - 16 * kt), at = d + (unsigned)(16 * kt), op = x + (unsigned)kt * step;
        tc_mma_f16_ts(at, op, hi, id, kt ? 1u : 0u);
        tc_mma_f16_ts(at, op, lo, id, 1u);
        tc_mma_f16_ts(at, op + 8, hi, id, 1u);
      }
    };
    for (; c < a.chunks; ++c) {
      const unsigned st = base + DS_STAGES_OFF + (unsigned)((c & 1) * DsStage::BYTES), ph = (unsigned)c & 1u;
      if (!hold(full(c & 1), (unsigned)(c >> 1) & 1u, 42) || !hold(sh_ready, ph, 43)) break;
      if (c > 0 && !hold(o_read, ph ^ 1u, 44)) break;
      if (lane == 0) {
        for (int ks = 0; ks < blocks; ++ks) {
          const unsigned long long x =
              umma_desc_k128(st + DsStage::KQ + (unsigned)((ks >> 2) * 2 * DS_BOX)) + (unsigned long long)((ks & 3) * 2);
          tc_mma_f16_ts(tmem + TM_PK, tmem + TM_SH + (unsigned)(ks * 16), x, id_p, ks ? 1u : 0u);
          tc_mma_f16_ts(tmem + TM_PK, tmem + TM_SH + (unsigned)(ks * 16 + 8), x, id_p, 1u);
        }
        tc_commit(p_full);
      }
      __syncwarp();
      if (!hold(r_ready, ph, 45)) break;
      if (lane == 0) {
        triangle(tmem + TM_U, tmem + TM_PK, 16, st + DsStage::MATS);
        tc_commit(u_full);
      }
      __syncwarp();
      if (!hold(uh_ready, ph, 46)) break;
      if (lane == 0) {
#pragma unroll
        for (int kt = 0; kt < 4; ++kt) {
          const unsigned long long x = umma_desc_mn128(st + DsStage::KQ + (unsigned)(kt * 2048), 2 * DS_BOX);
          tc_mma_f16_ts(tmem + TM_S, tmem + TM_UH + (unsigned)(kt * 32 + 16), x, id_s, 1u);
          tc_mma_f16_ts(tmem + TM_S, tmem + TM_UH + (unsigned)(kt * 32 + 24), x, id_s, 1u);
        }
        tc_commit(s_full);
        triangle(tmem + TM_UA, tmem + TM_UH, 32, st + DsStage::MATS + 2 * DS_BOX);
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
      if (!hold(full(c & 1), (unsigned)(c >> 1) & 1u, 48)) break;
      const float *fs = factors_of(c);
      const float keep = fs[3 * CH];
      if (c > 0 && !hold(s_full, ph ^ 1u, 49)) break;
      unsigned x[2][16];
#pragma unroll 1
      for (int k0 = half; k0 < blocks; k0 += 4) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int kt = k0 + 2 * i;
          if (kt >= blocks) break;
          if (c > 0) {
            tc_ld16(lanes + TM_S + (unsigned)(kt * 16), x[i]);
          } else {
#pragma unroll
            for (int j = 0; j < 16; ++j)
              x[i][j] = s.p0 > 0 && mine ? __float_as_uint(S[(long long)(kt * 16 + j) * a.vdim]) : 0u;
          }
        }
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int kt = k0 + 2 * i;
          if (kt >= blocks) break;
          float f[16];
          unsigned w[16];
#pragma unroll
          for (int j = 0; j < 16; ++j) f[j] = __uint_as_float(x[i][j]);
          operand_block<0>(f, w);
          tc_st16(lanes + TM_SH + (unsigned)(kt * 16), w);
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
      if (!hold(p_full, ph, 51)) break;
#pragma unroll
      for (int i = 0; i < 2; ++i) tc_ld16(lanes + TM_PK + (unsigned)((2 * i + half) * 16), x[i]);
      asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int kt = 2 * i + half;
        unsigned w[16];
#pragma unroll
        for (int j = 0; j < 16; j += 4) {
          const float4 y = *reinterpret_cast<const float4 *>(fs + kt * 16 + j);
          rhs[i][j] = fmaf(-y.x, __uint_as_float(x[i][j]), rhs[i][j]);
          rhs[i][j + 1] = fmaf(-y.y, __uint_as_float(x[i][j + 1]), rhs[i][j + 1]);
          rhs[i][j + 2] = fmaf(-y.z, __uint_as_float(x[i][j + 2]), rhs[i][j + 2]);
          rhs[i][j + 3] = fmaf(-y.w, __uint_as_float(x[i][j + 3]), rhs[i][j + 3]);
        }
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
        for (int j = 0; j < 16; j += 4) {
          const float4 y = *reinterpret_cast<const float4 *>(fs + 2 * CH + kt * 16 + j);
          f[j] *= y.x;
          f[j + 1] *= y.y;
          f[j + 2] *= y.z;
          f[j + 3] *= y.w;
        }
        operand_block<16>(f, w);
        tc_st32(lanes + TM_UH + (unsigned)(kt * 32), w);
      }
      release(uh_ready);
      if (lane == 0) mbar_arrive(empty(c & 1));
    }
    if (ok && hold(s_full, (unsigned)(a.chunks - 1) & 1u, 53)) {
#pragma unroll 1
      for (int kt = half; kt < blocks; kt += 2) {
        unsigned x[16];
        tc_ld16(lanes + TM_S + (unsigned)(kt * 16), x);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
        if (mine) {
#pragma unroll
          for (int j = 0; j < 16; ++j) S[(long long)(kt * 16 + j) * a.vdim] = __uint_as_float(x[j]);
        }
      }
    }
  } else {
    const int q = warp & 3, half = (warp - 2 - DS_CHAIN) >> 2, tid = threadIdx.x - (2 + DS_CHAIN) * 32;
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
    // whole rows of outputs: 16 lanes per token, eight columns each
    const int col = (tid & 15) * 8, row0 = tid >> 4;
    const bool in = col < vcols;
    const float inv_count = 1.0f / s.count;
    float w8[8] = {};
    if (s.normed && in) {
#pragma unroll
      for (int j = 0; j < 8; ++j) w8[j] = s.norm[col + j];
    }
    // the gates of this thread's eight pieces of a chunk, in its own corner of shared memory, a chunk ahead
    uint4 *gates = reinterpret_cast<uint4 *>(base_ptr + DS_GATE_OFF) + tid;
    auto fetch_gates = [&](int c) {
      if (s.normed) {
#pragma unroll
        for (int k = 0; k < DS_PIECES; ++k) {
          const int t = c * CH + row0 + k * (CH / DS_PIECES);
          const bool there = in && t < a.n;
          const bf16 *src = there ? s.gate + ((long long)b * a.n + t) * s.in_ld + h * a.vdim + col : s.gate;
          asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_u32(gates + k * DS_OUT * 32)), "l"(src),
                       "r"(there ? 16 : 0)
                       : "memory");
        }
      }
      asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch_gates(0);
    for (int c = 0; c < a.chunks && ok; ++c) {
      const unsigned ph = (unsigned)c & 1u;
      const int t0 = c * CH, nt = min(CH, a.n - t0);
      if (!hold(full(c & 1), (unsigned)(c >> 1) & 1u, 54) || !hold(o_full, ph, 55)) break;
      const float *fs = factors_of(c) + CH;
      {  // this warp's half of the tokens
        unsigned x[2][16], y[2][16];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          tc_ld16(lanes + TM_PQ + (unsigned)(half * 32 + i * 16), x[i]);
          tc_ld16(lanes + TM_UA + (unsigned)(half * 32 + i * 16), y[i]);
        }
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
        release(o_read);
        if (c > 0 && !hold(rows_out, ph ^ 1u, 56)) break;  // the last chunk's rows have been read
        float *to = staging + half * 32 * DS_SP + vl;
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
          for (int j = 0; j < 16; j += 4) {
            const float4 f = *reinterpret_cast<const float4 *>(fs + half * 32 + i * 16 + j);
            float *at = to + (i * 16 + j) * DS_SP;
            at[0] = vl < vcols ? fmaf(__uint_as_float(x[i][j]), f.x, __uint_as_float(y[i][j])) : 0.f;
            at[DS_SP] = vl < vcols ? fmaf(__uint_as_float(x[i][j + 1]), f.y, __uint_as_float(y[i][j + 1])) : 0.f;
            at[2 * DS_SP] = vl < vcols ? fmaf(__uint_as_float(x[i][j + 2]), f.z, __uint_as_float(y[i][j + 2])) : 0.f;
            at[3 * DS_SP] = vl < vcols ? fmaf(__uint_as_float(x[i][j + 3]), f.w, __uint_as_float(y[i][j + 3])) : 0.f;
          }
      }
      release(rows_in);
      if (lane == 0) mbar_arrive(empty(c & 1));
      if (!hold(rows_in, ph, 57)) break;
      asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll 1
      for (int k0 = 0; k0 < DS_PIECES; k0 += 4) {  // four rows together: their sums do not wait for one another
        float y[4][8], sum[4];
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const float *row = staging + (row0 + (CH / DS_PIECES) * (k0 + k)) * DS_SP + col;
          const float4 u = *reinterpret_cast<const float4 *>(row), w = *reinterpret_cast<const float4 *>(row + 4);
          const float e[8] = {u.x, u.y, u.z, u.w, w.x, w.y, w.z, w.w};
          float s0 = 0.f, s1 = 0.f;
#pragma unroll
          for (int j = 0; j < 8; j += 2) {
            y[k][j] = e[j];
            y[k][j + 1] = e[j + 1];
            s0 = fmaf(e[j], e[j], s0);
            s1 = fmaf(e[j + 1], e[j + 1], s1);
          }
          sum[k] = s0 + s1;
        }
        if (s.normed) {
#pragma unroll
          for (int o = 8; o > 0; o >>= 1)
#pragma unroll
            for (int k = 0; k < 4; ++k) sum[k] += __shfl_xor_sync(0xffffffffu, sum[k], o);
        }
#pragma unroll
        for (int k = 0; k < 4; ++k) {
          const int t = row0 + (CH / DS_PIECES) * (k0 + k);
          const long long r = (long long)b * a.n + t0 + t;
          const bool store = in && t < nt;
          if (!s.normed) {
            if (store) {
              float *o = s.o + (r * a.heads + h) * a.vdim + vt + col;
              *reinterpret_cast<float4 *>(o) = make_float4(y[k][0], y[k][1], y[k][2], y[k][3]);
              *reinterpret_cast<float4 *>(o + 4) = make_float4(y[k][4], y[k][5], y[k][6], y[k][7]);
            }
            continue;
          }
          const float inv = rsqrtf(sum[k] * inv_count + s.eps);
          const uint4 gate = gates[(k0 + k) * DS_OUT * 32];
          const unsigned g[4] = {gate.x, gate.y, gate.z, gate.w};
          unsigned out[4];
#pragma unroll
          for (int j = 0; j < 4; ++j)
            out[j] = pack2(y[k][2 * j] * inv * w8[2 * j] * silu_fast(lowf(g[j])),
                           y[k][2 * j + 1] * inv * w8[2 * j + 1] * silu_fast(highf(g[j])));
          if (store)
            *reinterpret_cast<uint4 *>(s.out + r * s.out_ld + h * a.vdim + col) = make_uint4(out[0], out[1], out[2], out[3]);
        }
      }
      release(rows_out);
      if (c + 1 < a.chunks) fetch_gates(c + 1);
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
