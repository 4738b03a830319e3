// Attention of many new rows on the sm_100a tensor cores (tcgen05 + TMEM + TMA), bfloat16 operands and
// 32-bit scores, weights and sums; a query sees the keys of its KeySpan (a sliding window or its chunk).
// Keys are row-major. Values come in one of two forms:
//   V_ROWS false   transposed (one row per value column, one column per key): a K-major operand as it
//                  lies; keys and values expanded from a window's latents
//   V_ROWS true    row-major like the keys, straight from a cache: an operand with its columns
//                  contiguous (64 columns per slab, eight keys per swizzle atom); query heads may share
//                  key and value heads
//
// One CTA per 128 queries of one head and stream walks the key tiles (128 keys) its rows see:
//   S = Q K^T      A = Q tile, B = K tile, into 128 columns of tensor memory
//   P              four warps, one thread per query row: maximum, weights 2^(s - m), stored as
//                  bfloat16 pairs over the scores' own columns (two keys per column)
//   O += P V       A = P from tensor memory, B = V tile
// The reference maximum of a row follows its running maximum only when that has grown by more than
// 2^8: until then the accumulated O and the sum stay as they are (weights up to 2^8 are exact enough
// in either format), so most tiles need no pass over O.
// Up to 128 value columns the CTA takes half of tensor memory and less than half of the shared
// memory: two CTAs share an SM, and one's products run under the other's softmax.
// Warp 0 issues TMA, warp 1 owns tensor memory and issues the MMAs. Every mbarrier wait is bounded; no
// clusters, no multicast.
#include "model.cuh"
#include "gemm_tc.cuh"
#include "tc_ptx.cuh"

#include <cuda_bf16.h>

namespace lb {

namespace {

typedef __nv_bfloat16 bf16;

constexpr int LP_BQ = 128, LP_BK = 128, LP_THREADS = 192;
constexpr int LP_SLAB = 128 * 128;  // 128 rows of 64 elements
constexpr float LP_NEG = -1.0e30f;
constexpr float LP_SLACK = 8.f;     // growth of a row's maximum that is left in the weights

__device__ __forceinline__ float lp_exp2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

struct LpArgs {
  int dim, vdim, n, n_rows;   // n new rows per stream
  int group;                  // query heads per key head
  int pos0;                   // position of a stream's first new row
  int first;                  // position of a stream's key row 0
  int key_base;               // key row 0 of stream 0 in the maps
  int key_rows, n_keys;       // key rows per stream as laid out, and those that exist
  KeySpan span;
  float factor;               // scale * log2(e)
  bf16 *out;
  int out_ld;
};

template <bool V_ROWS>
__global__ void __launch_bounds__(LP_THREADS, 2)
prefill_attention_kernel(const __grid_constant__ CUtensorMap map_q, const __grid_constant__ CUtensorMap map_k,
                      const __grid_constant__ CUtensorMap map_v, LpArgs a, DevErr *err) {
  extern __shared__ unsigned char smem_raw[];
  const unsigned base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  unsigned char *base_ptr = smem_raw + (base - smem_u32(smem_raw));
  const int dslabs = (a.dim + 63) >> 6;
  const unsigned q_off = base, k_off = base + (unsigned)(dslabs * LP_SLAB), v_off = k_off + (unsigned)(dslabs * LP_SLAB);
  // the V tile: two slabs of 64 keys by vdim rows, or slabs of 64 columns by 128 key rows
  const unsigned vslab = V_ROWS ? (unsigned)LP_SLAB : (unsigned)a.vdim * 128u;
  const int vslabs = V_ROWS ? (a.vdim + 63) >> 6 : 2;
  const unsigned bars = v_off + (unsigned)vslabs * vslab;
  unsigned char *bar_ptr = base_ptr + (bars - base);
  const unsigned q_full = bars, k_full = bars + 8, v_full = bars + 16, k_free = bars + 24, s_full = bars + 32,
                 p_ready = bars + 40, o_full = bars + 48;
  volatile unsigned *tmem_holder = reinterpret_cast<volatile unsigned *>(bar_ptr + 64);
  volatile int *abort_flag = reinterpret_cast<volatile int *>(bar_ptr + 68);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int h = blockIdx.y, b = blockIdx.z, t0 = blockIdx.x * LP_BQ;
  const unsigned cols = a.vdim <= 128 ? 256u : 512u;
  // key rows this tile of queries sees: [lo, hi]; lo rounded down to a 16-byte boundary of V^T's rows
  const int qrel0 = a.pos0 - a.first + t0;
  const int lo = max(0, a.span.first(a.pos0 + t0) - a.first) & ~(V_ROWS ? 0 : 7);
  const int kcol = h / a.group * a.dim, vcol = h / a.group * a.vdim, key0 = a.key_base + b * a.key_rows;
  const int hi = min(qrel0 + LP_BQ, a.n_keys) - 1;
  const int tiles = (hi - lo) / LP_BK + 1;

  if (threadIdx.x == 0) {
    for (unsigned bar : {q_full, k_full, v_full, k_free, s_full, o_full}) mbar_init(bar, 1);
    mbar_init(p_ready, 4);
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32((const void *)tmem_holder)),
                 "r"(cols)
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
  const unsigned tmem_s = *tmem_holder, tmem_o = tmem_s + LP_BK;
  pdl_launch_dependents();  // behind the allocation: a dependent's CTA must not take tensor memory first
  pdl_wait();

  if (warp == 0) {
    int k_loads = 0, v_loads = 0;
    bool ok = true;
    if (lane == 0) {
      mbar_expect_tx(q_full, (unsigned)(dslabs * LP_SLAB));
      for (int s = 0; s < dslabs; ++s) tma_load_2d(q_off + s * LP_SLAB, &map_q, h * a.dim + s * 64, b * a.n + t0, q_full);
    }
    for (int i = 0; i < tiles && ok; ++i) {
      const int j0 = lo + i * LP_BK;
      if (i > 0) ok = mbar_wait(k_free, (unsigned)(i - 1) & 1u, abort_flag, err, 21);
      __syncwarp();
      if (!ok) break;
      if (lane == 0) {
        mbar_expect_tx(k_full, (unsigned)(dslabs * LP_SLAB));
        for (int s = 0; s < dslabs; ++s)
          tma_load_2d(k_off + s * LP_SLAB, &map_k, kcol + s * 64, key0 + j0, k_full);
      }
      ++k_loads;
      if (i > 0) ok = mbar_wait(o_full, (unsigned)(i - 1) & 1u, abort_flag, err, 22);  // P V has read the V tile
      __syncwarp();
      if (!ok) break;
      if (lane == 0) {
        mbar_expect_tx(v_full, (unsigned)vslabs * vslab);
        for (int s = 0; s < vslabs; ++s) {
          if (V_ROWS) tma_load_2d(v_off + s * vslab, &map_v, vcol + s * 64, key0 + j0, v_full);
          else tma_load_2d(v_off + s * vslab, &map_v, key0 + j0 + s * 64, vcol, v_full);
        }
      }
      ++v_loads;
      __syncwarp();
    }
    if (*abort_flag) {  // copies in flight must land before the shared memory goes away
      const unsigned long long limit = global_timer() + WAIT_LIMIT_NS;
      while (!mbar_try_wait(q_full, 0) && global_timer() < limit) {}
      while (k_loads > 0 && !mbar_try_wait(k_full, (unsigned)(k_loads - 1) & 1u) && global_timer() < limit) {}
      while (v_loads > 0 && !mbar_try_wait(v_full, (unsigned)(v_loads - 1) & 1u) && global_timer() < limit) {}
    }
  } else if (warp == 1) {
    const unsigned idesc_s = umma_idesc_bf16(LP_BK), idesc_o = umma_idesc_bf16(a.vdim) | (V_ROWS ? UMMA_B_MN_MAJOR : 0u);
    const int ksteps = a.dim >> 4;
    bool ok = mbar_wait(q_full, 0, abort_flag, err, 23);
    __syncwarp();
    int i = 0;
    for (; i < tiles && ok; ++i) {
      ok = mbar_wait(k_full, (unsigned)i & 1u, abort_flag, err, 24);
      __syncwarp();
      if (!ok) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      if (lane == 0) {
        for (int ks = 0; ks < ksteps; ++ks) {
          const unsigned off = (unsigned)((ks >> 2) * LP_SLAB + (ks & 3) * 32);
          tc_mma_f16(tmem_s, umma_desc_k128(q_off + (unsigned)((ks >> 2) * LP_SLAB)) + (unsigned long long)((ks & 3) * 2),
                     umma_desc_k128(k_off + off - (unsigned)((ks & 3) * 32)) + (unsigned long long)((ks & 3) * 2), idesc_s,
                     ks ? 1u : 0u);
        }
        tc_commit(k_free);
        tc_commit(s_full);
      }
      __syncwarp();
      ok = mbar_wait(p_ready, (unsigned)i & 1u, abort_flag, err, 25);
      __syncwarp();
      if (!ok) break;
      ok = mbar_wait(v_full, (unsigned)i & 1u, abort_flag, err, 26);
      __syncwarp();
      if (!ok) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      if (lane == 0) {
#pragma unroll
        for (int ks = 0; ks < LP_BK / 16; ++ks)
          tc_mma_f16_ts(tmem_o, tmem_s + (unsigned)(ks * 8),
                        V_ROWS ? umma_desc_mn128(v_off + (unsigned)(ks * 16 * 128), vslab)
                               : umma_desc_k128(v_off + (unsigned)(ks >> 2) * vslab) + (unsigned long long)((ks & 3) * 2),
                        idesc_o, (i | ks) ? 1u : 0u);
        tc_commit(o_full);
      }
      __syncwarp();
    }
    if (!ok) {  // a bounded chance for the tensor pipe to finish before tensor memory is freed
      if (lane == 0) tc_commit(o_full);
      __syncwarp();
      const unsigned long long limit = global_timer() + WAIT_LIMIT_NS;
      while (!mbar_try_wait(o_full, (unsigned)i & 1u) && global_timer() < limit) {}
    }
  } else {
    const int q = warp & 3;
    const unsigned lanes = (unsigned)(q * 32) << 16;
    const int t = t0 + q * 32 + lane;     // this thread's row of the portion
    const int qrel = qrel0 + q * 32 + lane;  // its own key row
    const int row_lo = a.span.first(a.pos0 + t) - a.first, warp_lo = a.span.first(a.pos0 + t0 + q * 32 + 31) - a.first;
    const int wq0 = qrel0 + q * 32;       // the warp's first row
    float m = LP_NEG, l = 0.f;
    bool ok = true;
    for (int i = 0; i < tiles && ok; ++i) {
      const int j0 = lo + i * LP_BK;
      ok = mbar_wait_warp(s_full, (unsigned)i & 1u, abort_flag, err, 27);
      if (!ok) break;
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      // keys j0 + c seen by this row: c in [c_lo, c_hi]; whole tiles inside every row's span need no mask
      const int c_hi = qrel - j0, c_lo = row_lo - j0;
      const bool inside = wq0 - j0 >= LP_BK - 1 && warp_lo <= j0;
      // the row's scores stay in registers; independent chains for the maximum and the sum
      float s[LP_BK];
      {
        unsigned(&u)[4][32] = reinterpret_cast<unsigned(&)[4][32]>(s);
#pragma unroll
        for (int c = 0; c < 4; ++c) tc_ld32(tmem_s + lanes + (unsigned)(c * 32), u[c]);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
      }
#pragma unroll
      for (int j = 0; j < LP_BK; ++j) s[j] *= a.factor;
      if (!inside) {
#pragma unroll
        for (int j = 0; j < LP_BK; ++j)
          if (j > c_hi || j < c_lo) s[j] = 2.f * LP_NEG;  // weight zero against any reference maximum
      }
      float mq[4] = {s[0], s[1], s[2], s[3]};
#pragma unroll
      for (int j = 4; j < LP_BK; ++j) mq[j & 3] = fmaxf(mq[j & 3], s[j]);
      const float mx = fmaxf(LP_NEG, fmaxf(fmaxf(mq[0], mq[1]), fmaxf(mq[2], mq[3])));
      const bool grow = mx > m + LP_SLACK;
      const float keep = grow ? lp_exp2(m - mx) : 1.f;
      if (grow) m = mx;
      l *= keep;
      if (i > 0) {
        ok = mbar_wait_warp(o_full, (unsigned)(i - 1) & 1u, abort_flag, err, 28);
        if (!ok) break;
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        if (__any_sync(0xffffffffu, grow)) {
#pragma unroll 1
          for (int c0 = 0; c0 < a.vdim; c0 += 16) {
            unsigned r[16];
            tc_ld16(tmem_o + lanes + (unsigned)c0, r);
            asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
#pragma unroll
            for (int j = 0; j < 16; ++j) r[j] = __float_as_uint(__uint_as_float(r[j]) * keep);
            tc_st16(tmem_o + lanes + (unsigned)c0, r);
          }
        }
      }
      float lq[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int c0 = 0; c0 < LP_BK; c0 += 32) {
        unsigned pk[16];
#pragma unroll
        for (int j = 0; j < 32; j += 2) {
          const float e0 = lp_exp2(s[c0 + j] - m), e1 = lp_exp2(s[c0 + j + 1] - m);
          lq[j & 2] += e0;
          lq[(j & 2) + 1] += e1;
          const __nv_bfloat162 v = __floats2bfloat162_rn(e0, e1);
          pk[j >> 1] = *reinterpret_cast<const unsigned *>(&v);
        }
        tc_st16(tmem_s + lanes + (unsigned)(c0 >> 1), pk);  // over the scores, which this warp has read
      }
      l += (lq[0] + lq[1]) + (lq[2] + lq[3]);
      asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
      __syncwarp();
      if (lane == 0) mbar_arrive(p_ready);
    }
    if (ok) ok = mbar_wait_warp(o_full, (unsigned)(tiles - 1) & 1u, abort_flag, err, 29);
    if (ok) {
      asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
      const float inv = 1.0f / l;
      bf16 *o = a.out + ((long long)b * a.n + t) * a.out_ld + (long long)h * a.vdim;
#pragma unroll 1
      for (int c0 = 0; c0 < a.vdim; c0 += 16) {
        unsigned r[16];
        tc_ld16(tmem_o + lanes + (unsigned)c0, r);
        asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
        unsigned pk[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          const __nv_bfloat162 v = __floats2bfloat162_rn(__uint_as_float(r[2 * j]) * inv, __uint_as_float(r[2 * j + 1]) * inv);
          pk[j] = *reinterpret_cast<const unsigned *>(&v);
        }
        if (t < a.n) {
          *reinterpret_cast<uint4 *>(o + c0) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
          *reinterpret_cast<uint4 *>(o + c0 + 8) = make_uint4(pk[4], pk[5], pk[6], pk[7]);
        }
      }
    }
  }
  __syncwarp();
  asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
  __syncthreads();
  if (warp == 1) {
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_s), "r"(cols));
  }
}

size_t lp_smem(int dim, int vdim, bool v_rows) {
  return (size_t)2 * ((dim + 63) / 64) * LP_SLAB + (v_rows ? (size_t)((vdim + 63) / 64) * LP_SLAB : (size_t)2 * vdim * 128) +
         128 + 1024;
}

bool lp_sizes(int dim, int vdim) {
  return dim % 16 == 0 && vdim % 16 == 0 && dim >= 16 && vdim >= 16 && dim <= 256 && vdim <= 256;
}

template <bool V_ROWS>
void lp_launch(const CUtensorMap &mq, const CUtensorMap &mk, const CUtensorMap &mv, const LpArgs &a, int heads, int streams,
               cudaStream_t st, DevErr *err) {
  const size_t smem = lp_smem(a.dim, a.vdim, V_ROWS);
  LB_CUDA(cudaFuncSetAttribute(prefill_attention_kernel<V_ROWS>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  launch_pdl(prefill_attention_kernel<V_ROWS>, dim3((unsigned)((a.n + LP_BQ - 1) / LP_BQ), (unsigned)heads, (unsigned)streams),
             dim3(LP_THREADS), smem, st, false, mq, mk, mv, a, err);
}

}  // namespace

bool latent_prefill_supports(int dim, int vdim) { return lp_sizes(dim, vdim); }
bool grouped_prefill_supports(int dim, int vdim) { return lp_sizes(dim, vdim); }

void launch_latent_prefill(const LatentAttention &at, const void *k, int k_ld, const void *vt, int vt_ld, int key_rows,
                           int first, const RowBatch &b, cudaStream_t st, DevErr *err) {
  LpArgs a{};
  a.dim = at.dim;
  a.vdim = at.vdim;
  a.n = b.n;
  a.group = 1;
  a.pos0 = b.p0;
  a.first = first;
  a.key_rows = key_rows;
  a.n_keys = b.p0 + b.n - first;
  a.span.size = at.window;
  a.factor = at.scale * 1.4426950408889634f;
  a.out = static_cast<bf16 *>(at.out);
  a.out_ld = at.out_ld;
  CUtensorMap mq, mk, mv;
  const unsigned long long hd = (unsigned long long)at.heads * at.dim, hv = (unsigned long long)at.heads * at.vdim;
  const unsigned long long keys = (unsigned long long)b.streams * key_rows;
  tc_make_map_bf16(&mq, at.q, (unsigned long long)b.rows(), hd, (unsigned long long)at.q_ld, LP_BQ);
  tc_make_map_bf16(&mk, k, keys, hd, (unsigned long long)k_ld, LP_BK);
  tc_make_map_bf16(&mv, vt, hv, keys, (unsigned long long)vt_ld, (unsigned)at.vdim);
  lp_launch<false>(mq, mk, mv, a, at.heads, b.streams, st, err);
}

void launch_grouped_prefill(const GroupedAttention &at, const RowBatch &b, cudaStream_t st, DevErr *err) {
  LpArgs a{};
  a.dim = at.dim;
  a.vdim = at.vdim;
  a.n = b.n;
  a.group = at.heads / at.groups;
  a.pos0 = b.p0;
  a.key_base = b.slot0 * at.cap;
  a.key_rows = at.cap;
  a.n_keys = b.p0 + b.n;
  a.span = at.span;
  a.factor = at.scale * 1.4426950408889634f;
  a.out = static_cast<bf16 *>(at.out);
  a.out_ld = at.out_ld;
  CUtensorMap mq, mk, mv;
  const unsigned long long kd = (unsigned long long)at.groups * at.dim, vd = (unsigned long long)at.groups * at.vdim;
  const unsigned long long keys = (unsigned long long)at.slots * at.cap;
  tc_make_map_bf16(&mq, at.q, (unsigned long long)b.rows(), (unsigned long long)at.heads * at.dim, (unsigned long long)at.q_ld,
                   LP_BQ);
  tc_make_map_bf16(&mk, at.k_cache, keys, kd, kd, LP_BK);
  tc_make_map_bf16(&mv, at.v_cache, keys, vd, vd, LP_BK);
  lp_launch<true>(mq, mk, mv, a, at.heads, b.streams, st, err);
}

}  // namespace lb
