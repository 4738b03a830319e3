// The gated delta rule of many new rows on bfloat16, in chunks of 64 tokens.
//
// Inside a chunk, with G_i the sum of the logarithms of the decays up to token i, r_i = 1 / |k'_i|,
// r'_i = dim^-1/2 / |q'_i| (k', q' the convolved vectors as stored) and S the state before the chunk, the rule's
// updates u_i solve a unit lower triangular system:
//   L_ij = beta_i r_i r_j e^(G_i - G_j) (k'_i . k'_j)  (j < i),   (I + L) U = diag(beta) (V - diag(e^G_i r_i) K' S)
//   A_ij = r'_i r_j e^(G_i - G_j) (q'_i . k'_j)        (j <= i),  O = diag(e^G_i r'_i) Q' S + A U
//   S <- e^G_last S + (diag(e^(G_last - G_j) r_j) K')^T U
// Exponents are never positive, and the vectors' norms stay out of the matrix operands, which are the stored
// bfloat16 values themselves. Everything else that enters a product (the state, (I + L)^-1 diag(beta), A, the
// right-hand side, U) is 32-bit and enters as two bfloat16 terms.
//
//   delta_prepare_kernel   per chunk and head: Q'K'^T and A, K'K'^T and L, the inverse by blocks of 32, and the
//                          factors of a token; no chunk depends on another
//   delta_scan_kernel      per stream, head and tile of value columns: the chunks in order, for the sizes that
//                          delta_scan_tc.cu leaves (few value columns, heads beyond 128). A warp owns 16 value columns
//                          and keeps their part of S^T in registers as accumulators of mma.sync tiles, whose layout is
//                          that of the next product's left operand: the chain S^T K'^T -> right-hand side -> U^T ->
//                          O^T, S^T runs without leaving the warp, on tiles of K', Q', V and the chunk's matrices that
//                          all warps share (cp.async, two stages). Where the CTA holds a whole head the output's norm
//                          and gate follow at once.
#include "delta.cuh"

namespace lb {

namespace {

typedef __nv_bfloat16 bf16;

constexpr int CH = DELTA_CHUNK;
constexpr int MP = CH + 8;       // pitch of the chunk's matrices in shared memory
constexpr int PREP_THREADS = 128;
constexpr int TP = 68;           // pitch of the float matrices

__device__ __forceinline__ unsigned smem_addr(const void *p) { return (unsigned)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldmatrix4(unsigned (&r)[4], const bf16 *p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_addr(p)));
}
__device__ __forceinline__ void ldmatrix4_trans(unsigned (&r)[4], const bf16 *p) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3])
               : "r"(smem_addr(p)));
}
// (Not volatile: a function of registers, the compiler may spread them between the loads.)
__device__ __forceinline__ void mma(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// 16 bytes to shared memory in the background; false stores zeros.
__device__ __forceinline__ void copy16(void *dst, const void *src, bool in) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(in ? 16 : 0) : "memory");
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void copy_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }

__device__ __forceinline__ unsigned pack(float a, float b) {
  const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const unsigned *>(&v);
}
__device__ __forceinline__ float low_half(unsigned u) { return __uint_as_float(u << 16); }
__device__ __forceinline__ float high_half(unsigned u) { return __uint_as_float(u & 0xffff0000u); }
// Two floats as two terms of two packed bfloat16 each.
__device__ __forceinline__ void split(float a, float b, unsigned &hi, unsigned &lo) {
  hi = pack(a, b);
  lo = pack(a - low_half(hi), b - high_half(hi));
}
// Left operand (16 x 16) from two neighbouring accumulator tiles of 16 x 8.
__device__ __forceinline__ void operand(const float (&c0)[4], const float (&c1)[4], unsigned (&hi)[4], unsigned (&lo)[4]) {
  split(c0[0], c0[1], hi[0], lo[0]);
  split(c0[2], c0[3], hi[1], lo[1]);
  split(c1[0], c1[1], hi[2], lo[2]);
  split(c1[2], c1[3], hi[3], lo[3]);
}

// acc += a x over the right operand's blocks of 16 rows from the given one on.
__device__ __forceinline__ void terms(float (&acc)[8][4], const unsigned (&a)[4], const unsigned (&x)[4][4], int from = 0) {
#pragma unroll
  for (int j = 0; j < 4; ++j)
    if (j >= from) {
      mma(acc[2 * j], a, x[j][0], x[j][1]);
      mma(acc[2 * j + 1], a, x[j][2], x[j][3]);
    }
}

constexpr double LOG2E = 1.4426950408889634;
__device__ __forceinline__ float exp2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// Difference of two numbers in two terms each.
__device__ __forceinline__ float apart(float2 a, float2 b) { return (a.x - b.x) + (a.y - b.y); }

struct PrepareArgs {
  DeltaChunks c;
  float q_scale;
  const float *a_log, *dt_bias;
  const float *ba;
  int ba_ld;
};

// Of a chunk's matrices only blocks of 16 columns that start at or below the diagonal of their 16 rows are written and read.
constexpr int MAT = CH * CH;
__device__ __forceinline__ long long chunk_at(const DeltaChunks &a, int b, int h, int chunk) {
  return ((long long)b * a.heads + h) * a.chunks + chunk;
}

__global__ void __launch_bounds__(PREP_THREADS, 5)
delta_prepare_kernel(PrepareArgs p) {
  const DeltaChunks &a = p.c;
  extern __shared__ __align__(16) unsigned char raw[];
  const int pitch = a.dim + 8;
  bf16 *ks = reinterpret_cast<bf16 *>(raw), *qs = ks + CH * pitch;
  float *lt = reinterpret_cast<float *>(raw);  // [64][TP] L transposed, over the vectors once the products are done
  float *ts = lt + CH * TP;                    // [64][TP] its inverse
  __shared__ float2 gs[CH];  // sums of the decays' logarithms to base 2, in two terms
  __shared__ float rk[CH], rq[CH], bs[CH];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, wid = tid >> 5, g = lane >> 2, t2 = (lane & 3) * 2;
  const int chunk = blockIdx.x, h = blockIdx.y, b = blockIdx.z, grp = h / (a.heads / a.groups);
  const int t0 = chunk * CH, nt = min(CH, a.n - t0);
  const long long r0 = (long long)b * a.n + t0;
  const bf16 *src = a.conv + r0 * a.channels + grp * a.dim;
  const int pieces = a.dim >> 3;
  for (int i = tid; i < CH * pieces; i += PREP_THREADS) {
    const int t = i / pieces, c = (i - t * pieces) * 8;
    const bf16 *row = t < nt ? src + (long long)t * a.channels + c : src;
    copy16(qs + t * pitch + c, row, t < nt);
    copy16(ks + t * pitch + c, row + a.groups * a.dim, t < nt);
  }
  copy_commit();
  if (wid == 0) {  // sums of the decays' logarithms, two tokens per lane
    double x[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int t = lane * 2 + i;
      const float *row = p.ba + (r0 + t) * p.ba_ld + h;
      x[i] = t < nt ? (double)delta_log_decay(row[a.heads], p.a_log[h], p.dt_bias[h]) : 0.0;
      bs[t] = t < nt ? sigmoid_f32(row[0]) : 0.f;
    }
    double sum = x[0] + x[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const double y = __shfl_up_sync(0xffffffffu, sum, o);
      if (lane >= o) sum += y;
    }
    auto two = [](double v) {
      const float hi = (float)v;
      return make_float2(hi, (float)(v - (double)hi));
    };
    gs[lane * 2] = two((sum - x[1]) * LOG2E);
    gs[lane * 2 + 1] = two(sum * LOG2E);
  }
  copy_wait_all();
  __syncthreads();
  const long long at = chunk_at(a, b, h, chunk);
  // products of the warp's 16 rows with the tokens up to its last row
  const int w0 = wid * 16;
  const int ar = w0 + (lane & 15), ac = (lane >> 4) * 8;                        // left operand's row and column
  const int br = (lane & 7) + ((lane >> 4) << 3), bc = ((lane >> 3) & 1) * 8;  // right operand: two tiles of 8 tokens
  {  // squares of the vectors' norms: the diagonals of the warp's own 16 by 16 blocks
    float dk[2][4] = {}, dq[2][4] = {};
#pragma unroll 2
    for (int c = 0; c < a.dim; c += 16) {
      unsigned x[4], y[4];
      ldmatrix4(x, ks + ar * pitch + c + ac);
      ldmatrix4(y, ks + (w0 + br) * pitch + c + bc);
      mma(dk[0], x, y[0], y[1]);
      mma(dk[1], x, y[2], y[3]);
      ldmatrix4(x, qs + ar * pitch + c + ac);
      ldmatrix4(y, qs + (w0 + br) * pitch + c + bc);
      mma(dq[0], x, y[0], y[1]);
      mma(dq[1], x, y[2], y[3]);
    }
    if ((g >> 1) == (lane & 3)) {
      const bool odd = g & 1;
      rk[w0 + g] = 1.0f / sqrtf((odd ? dk[0][1] : dk[0][0]) + DELTA_UNIT_EPS);
      rk[w0 + g + 8] = 1.0f / sqrtf((odd ? dk[1][3] : dk[1][2]) + DELTA_UNIT_EPS);
      rq[w0 + g] = p.q_scale / sqrtf((odd ? dq[0][1] : dq[0][0]) + DELTA_UNIT_EPS);
      rq[w0 + g + 8] = p.q_scale / sqrtf((odd ? dq[1][3] : dq[1][2]) + DELTA_UNIT_EPS);
    }
  }
  __syncthreads();
  if (tid < CH) {
    const float2 last = gs[CH - 1];
    const float e = exp2_fast(gs[tid].x);
    float *f = a.factors + at * 4 * CH + tid;
    f[0] = e * rk[tid];
    f[CH] = e * rq[tid];
    f[2 * CH] = exp2_fast(apart(last, gs[tid])) * rk[tid];
    f[3 * CH] = exp2_fast(last.x);
  }
  bf16 *mat = a.mats + at * 4 * MAT;
  float acc[8][4];
  auto product = [&](const bf16 *left) {
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[i][j] = 0.f;
#pragma unroll 2
    for (int c = 0; c < a.dim; c += 16) {
      unsigned x[4];
      ldmatrix4(x, left + ar * pitch + c + ac);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        if (j <= wid) {
          unsigned y[4];
          ldmatrix4(y, ks + (j * 16 + br) * pitch + c + bc);
          mma(acc[2 * j], x, y[0], y[1]);
          mma(acc[2 * j + 1], x, y[2], y[3]);
        }
      }
    }
  };
  const float2 gi[2] = {gs[w0 + g], gs[w0 + g + 8]};
  const float ri[2] = {rk[w0 + g] * bs[w0 + g], rk[w0 + g + 8] * bs[w0 + g + 8]}, qi[2] = {rq[w0 + g], rq[w0 + g + 8]};
  product(qs);
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    if (j <= 2 * wid + 1) {
      const int col = j * 8 + t2;
      const float2 g0 = gs[col], g1 = gs[col + 1];
      const float r0k = rk[col], r1k = rk[col + 1];
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int i = w0 + g + half * 8;
        const float v0 = col <= i ? exp2_fast(apart(gi[half], g0)) * r0k * qi[half] * acc[j][half * 2] : 0.f;
        const float v1 = col + 1 <= i ? exp2_fast(apart(gi[half], g1)) * r1k * qi[half] * acc[j][half * 2 + 1] : 0.f;
        unsigned hi, lo;
        split(v0, v1, hi, lo);
        *reinterpret_cast<unsigned *>(mat + 2 * MAT + i * CH + col) = hi;
        *reinterpret_cast<unsigned *>(mat + 3 * MAT + i * CH + col) = lo;
      }
    }
  }
  product(ks);
  __syncthreads();  // the vectors are read
#pragma unroll
  for (int j = 0; j < 8; ++j) {
    if (j <= 2 * wid + 1) {
#pragma unroll
      for (int k = 0; k < 2; ++k) {
        const int col = j * 8 + t2 + k;
        const float2 gc = gs[col];
        const float rc = rk[col];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int i = w0 + g + half * 8;
          lt[col * TP + i] = col < i ? exp2_fast(apart(gi[half], gc)) * rc * ri[half] * acc[j][half * 2 + k] : 0.f;
        }
      }
    }
  }
  __syncthreads();
  // inverse of I + L: the two diagonal blocks of 32 by substitution, one column per lane; a solved entry is taken out of
  // all later ones at once
  if (wid < 2) {
    const float *lb = lt + wid * 32 * TP + wid * 32;
    float x[32];
#pragma unroll
    for (int i = 0; i < 32; ++i) x[i] = i == lane ? 1.f : 0.f;
#pragma unroll
    for (int j = 0; j < 31; ++j) {
#pragma unroll
      for (int i = j / 4 * 4; i < 32; i += 4) {
        const float4 l = *reinterpret_cast<const float4 *>(lb + j * TP + i);
        if (i > j) x[i] = fmaf(-l.x, x[j], x[i]);
        if (i + 1 > j) x[i + 1] = fmaf(-l.y, x[j], x[i + 1]);
        if (i + 2 > j) x[i + 2] = fmaf(-l.z, x[j], x[i + 2]);
        if (i + 3 > j) x[i + 3] = fmaf(-l.w, x[j], x[i + 3]);
      }
    }
#pragma unroll
    for (int i = 0; i < 32; ++i) ts[(wid * 32 + i) * TP + wid * 32 + lane] = x[i];
  }
  __syncthreads();
  {  // the block below them: -(second inverse) L21 (first inverse); the upper right block holds L21 (first inverse)
    const int r = tid >> 2, c = (tid & 3) * 8;
    float m[8] = {};
#pragma unroll 8
    for (int j = 0; j < 32; ++j) {
      const float l = lt[j * TP + 32 + r];
      const float4 x = *reinterpret_cast<const float4 *>(ts + j * TP + c), y = *reinterpret_cast<const float4 *>(ts + j * TP + c + 4);
      m[0] = fmaf(l, x.x, m[0]);
      m[1] = fmaf(l, x.y, m[1]);
      m[2] = fmaf(l, x.z, m[2]);
      m[3] = fmaf(l, x.w, m[3]);
      m[4] = fmaf(l, y.x, m[4]);
      m[5] = fmaf(l, y.y, m[5]);
      m[6] = fmaf(l, y.z, m[6]);
      m[7] = fmaf(l, y.w, m[7]);
    }
    *reinterpret_cast<float4 *>(ts + r * TP + 32 + c) = make_float4(m[0], m[1], m[2], m[3]);
    *reinterpret_cast<float4 *>(ts + r * TP + 32 + c + 4) = make_float4(m[4], m[5], m[6], m[7]);
    __syncthreads();
    float n[8] = {};
#pragma unroll 8
    for (int j = 0; j < 32; ++j) {
      const float l = -ts[(32 + r) * TP + 32 + j];
      const float *row = ts + j * TP + 32 + c;
      const float4 x = *reinterpret_cast<const float4 *>(row), y = *reinterpret_cast<const float4 *>(row + 4);
      n[0] = fmaf(l, x.x, n[0]);
      n[1] = fmaf(l, x.y, n[1]);
      n[2] = fmaf(l, x.z, n[2]);
      n[3] = fmaf(l, x.w, n[3]);
      n[4] = fmaf(l, y.x, n[4]);
      n[5] = fmaf(l, y.y, n[5]);
      n[6] = fmaf(l, y.z, n[6]);
      n[7] = fmaf(l, y.w, n[7]);
    }
    *reinterpret_cast<float4 *>(ts + (32 + r) * TP + c) = make_float4(n[0], n[1], n[2], n[3]);
    *reinterpret_cast<float4 *>(ts + (32 + r) * TP + c + 4) = make_float4(n[4], n[5], n[6], n[7]);
  }
  __syncthreads();
  for (int i = tid; i < CH * (CH / 8); i += PREP_THREADS) {
    const int r = i >> 3, c = (i & 7) * 8;
    if (c >= (r / 16 + 1) * 16) continue;
    const float *row = ts + r * TP + c;
    const float4 x = *reinterpret_cast<const float4 *>(row), y = *reinterpret_cast<const float4 *>(row + 4);
    const float e[8] = {x.x, x.y, x.z, x.w, y.x, y.y, y.z, y.w};
    unsigned hi[4], lo[4];
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const int c0 = c + 2 * k, c1 = c0 + 1;
      split(c0 <= r ? e[2 * k] * bs[c0] : 0.f, c1 <= r ? e[2 * k + 1] * bs[c1] : 0.f, hi[k], lo[k]);
    }
    *reinterpret_cast<uint4 *>(mat + r * CH + c) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
    *reinterpret_cast<uint4 *>(mat + MAT + r * CH + c) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
  }
}

struct ScanArgs {
  DeltaChunks c;
  int p0, slot0, stages;
  float *state, *o;
  const bf16 *gate;
  int in_ld, out_ld, normed;
  float count, eps;
  const float *norm;
  bf16 *out;
};

// Shared memory of a stage, in bfloat16 elements (the token factors, 256 floats, behind them).
__host__ __device__ __forceinline__ int stage_elems(int dim, int vt) {
  return 2 * CH * (dim + 8) + CH * (vt + 8) + 4 * CH * MP + CH * 8;
}

// NT: tiles of 8 state rows (dim / 8 at most); WARPS: 16 value columns each. TWO_PASS: the products of the state
// with keys and with queries one after the other (fewer registers).
template <int NT, int WARPS, bool TWO_PASS>
__global__ void __launch_bounds__(WARPS * 32)
delta_scan_kernel(ScanArgs s) {
  constexpr int THREADS = WARPS * 32, VT = WARPS * 16, SP = VT + 4;
  extern __shared__ __align__(16) unsigned char raw[];
  const DeltaChunks &a = s.c;
  const int pitch = a.dim + 8, vp = VT + 8, elems = stage_elems(a.dim, VT);
  bf16 *stages = reinterpret_cast<bf16 *>(raw);
  float *stage_o = reinterpret_cast<float *>(stages + (size_t)s.stages * elems);  // [64][SP] outputs of the chunk
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, wid = tid >> 5, g = lane >> 2, t2 = (lane & 3) * 2;
  const int tiles = (a.vdim + VT - 1) / VT;
  const int h = blockIdx.x / tiles, vt = (blockIdx.x - h * tiles) * VT, b = blockIdx.y;
  const int grp = h / (a.heads / a.groups);
  const int cols = min(VT, a.vdim - vt);
  const bf16 *base = a.conv + (long long)b * a.n * a.channels;
  const int q_at = grp * a.dim, k_at = (a.groups + grp) * a.dim, v_at = 2 * a.groups * a.dim + h * a.vdim + vt;
  auto load = [&](int chunk) {
    bf16 *ks = stages + (size_t)(chunk % s.stages) * elems, *qs = ks + CH * pitch, *vs = qs + CH * pitch, *ms = vs + CH * vp;
    float *fs = reinterpret_cast<float *>(ms + 4 * CH * MP);
    const int t0 = chunk * CH, nt = min(CH, a.n - t0), pieces = a.dim >> 3;
    const bf16 *rows = base + (long long)t0 * a.channels;
    for (int i = tid; i < CH * pieces; i += THREADS) {
      const int t = i / pieces, c = (i - t * pieces) * 8;
      const bf16 *row = t < nt ? rows + (long long)t * a.channels : rows;
      copy16(ks + t * pitch + c, row + k_at + c, t < nt);
      copy16(qs + t * pitch + c, row + q_at + c, t < nt);
    }
    for (int i = tid; i < CH * (VT / 8); i += THREADS) {
      const int t = i / (VT / 8), c = (i - t * (VT / 8)) * 8;
      const bool in = t < nt && c < cols;
      copy16(vs + t * vp + c, in ? rows + (long long)t * a.channels + v_at + c : rows, in);
    }
    const long long at = chunk_at(a, b, h, chunk);
    for (int i = tid; i < 4 * CH * 8; i += THREADS) {
      const int m = i >> 9, r = (i >> 3) & 63, c = (i & 7) * 8;
      if (c < (r / 16 + 1) * 16) copy16(ms + (m * CH + r) * MP + c, a.mats + (at * 4 + m) * MAT + r * CH + c, true);
    }
    for (int i = tid * 4; i < 4 * CH; i += THREADS * 4) copy16(fs + i, a.factors + at * 4 * CH + i, true);
    copy_commit();
  };
  load(0);
  // S^T: this warp's 16 value columns by all state rows; element (v, d) of tile d / 8
  const int v0 = vt + wid * 16 + g;
  float *S = s.state + ((long long)(s.slot0 + b) * a.heads + h) * a.dim * a.vdim;
  float st[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int d = i * 8 + t2 + (j & 1), v = v0 + (j >> 1) * 8;
      st[i][j] = s.p0 > 0 && d < a.dim && v < a.vdim ? S[(long long)d * a.vdim + v] : 0.f;
    }
  const int br = (lane & 7) + ((lane >> 4) << 3), bc = ((lane >> 3) & 1) * 8;  // right operand, index rows
  const int tr = (lane & 7) + ((lane >> 3) & 1) * 8, tc = (lane >> 4) * 8;     // right operand, k rows (transposed on load)
  for (int chunk = 0; chunk < a.chunks; ++chunk) {
    copy_wait_all();
    __syncthreads();
    if (s.stages > 1 && chunk + 1 < a.chunks) load(chunk + 1);
    const bf16 *ks = stages + (size_t)(chunk % s.stages) * elems, *qs = ks + CH * pitch, *vs = qs + CH * pitch,
               *ms = vs + CH * vp;
    const float *fs = reinterpret_cast<const float *>(ms + 4 * CH * MP);
    float pk[8][4], pq[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) pk[i][j] = pq[i][j] = 0.f;
    // S^T K'^T (and S^T Q'^T)
#pragma unroll
    for (int kt = 0; kt < NT / 2; ++kt) {
      if (kt * 16 < a.dim) {
        unsigned hi[4], lo[4], x[4][4], y[4][4];
        operand(st[2 * kt], st[2 * kt + 1], hi, lo);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          ldmatrix4(x[j], ks + (j * 16 + br) * pitch + kt * 16 + bc);
          if (!TWO_PASS) ldmatrix4(y[j], qs + (j * 16 + br) * pitch + kt * 16 + bc);
        }
        terms(pk, lo, x);  // products that add to one accumulator stand far apart
        if (!TWO_PASS) terms(pq, lo, y);
        terms(pk, hi, x);
        if (!TWO_PASS) terms(pq, hi, y);
      }
    }
    // right-hand side V^T - e^G r (S^T K'^T)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      unsigned x[4];
      ldmatrix4_trans(x, vs + (j * 16 + br) * vp + wid * 16 + bc);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = j * 16 + i * 8 + t2;
        const float f0 = fs[t], f1 = fs[t + 1];
        float(&p)[4] = pk[2 * j + i];
        p[0] = low_half(x[2 * i]) - f0 * p[0];
        p[1] = high_half(x[2 * i]) - f1 * p[1];
        p[2] = low_half(x[2 * i + 1]) - f0 * p[2];
        p[3] = high_half(x[2 * i + 1]) - f1 * p[3];
      }
    }
    // U^T = (right-hand side)^T ((I + L)^-1 diag(beta))^T
    float u[8][4];
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) u[i][j] = 0.f;
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      unsigned hi[4], lo[4], x[4][4], y[4][4];
      operand(pk[2 * kt], pk[2 * kt + 1], hi, lo);
#pragma unroll
      for (int j = kt; j < 4; ++j) {
        ldmatrix4(x[j], ms + (j * 16 + br) * MP + kt * 16 + bc);
        ldmatrix4(y[j], ms + (CH + j * 16 + br) * MP + kt * 16 + bc);
      }
      terms(u, lo, x, kt);
      terms(u, hi, y, kt);
      terms(u, hi, x, kt);
    }
    if (TWO_PASS) {
#pragma unroll
      for (int kt = 0; kt < NT / 2; ++kt) {
        if (kt * 16 < a.dim) {
          unsigned hi[4], lo[4], x[4][4];
          operand(st[2 * kt], st[2 * kt + 1], hi, lo);
#pragma unroll
          for (int j = 0; j < 4; ++j) ldmatrix4(x[j], qs + (j * 16 + br) * pitch + kt * 16 + bc);
          terms(pq, lo, x);
          terms(pq, hi, x);
        }
      }
    }
    // O^T = e^G r' (S^T Q'^T) + U^T A^T
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const float f0 = fs[CH + i * 8 + t2], f1 = fs[CH + i * 8 + t2 + 1];
      pq[i][0] *= f0;
      pq[i][1] *= f1;
      pq[i][2] *= f0;
      pq[i][3] *= f1;
    }
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
      unsigned hi[4], lo[4], x[4][4], y[4][4];
      operand(u[2 * kt], u[2 * kt + 1], hi, lo);
#pragma unroll
      for (int j = kt; j < 4; ++j) {
        ldmatrix4(x[j], ms + (2 * CH + j * 16 + br) * MP + kt * 16 + bc);
        ldmatrix4(y[j], ms + (3 * CH + j * 16 + br) * MP + kt * 16 + bc);
      }
      terms(pq, lo, x, kt);
      terms(pq, hi, y, kt);
      terms(pq, hi, x, kt);
    }
    // S^T <- e^G_last S^T + (U^T diag(e^(G_last - G) r)) K'
    const float keep = fs[3 * CH];
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) st[i][j] *= keep;
#pragma unroll
    for (int kt = 0; kt < 4; ++kt) {
#pragma unroll
      for (int i = 2 * kt; i < 2 * kt + 2; ++i) {
        const float f0 = fs[2 * CH + i * 8 + t2], f1 = fs[2 * CH + i * 8 + t2 + 1];
        u[i][0] *= f0;
        u[i][1] *= f1;
        u[i][2] *= f0;
        u[i][3] *= f1;
      }
      unsigned hi[4], lo[4];
      operand(u[2 * kt], u[2 * kt + 1], hi, lo);
#pragma unroll
      for (int i = 0; i < NT / 2; i += 4) {
        unsigned x[4][4];
#pragma unroll
        for (int j = 0; j < 4; ++j)
          if ((i + j) * 16 < a.dim) ldmatrix4_trans(x[j], ks + (kt * 16 + tr) * pitch + (i + j) * 16 + tc);
#pragma unroll
        for (int term = 0; term < 2; ++term)
#pragma unroll
          for (int j = 0; j < 4; ++j)
            if ((i + j) * 16 < a.dim) {
              mma(st[2 * (i + j)], term ? hi : lo, x[j][0], x[j][1]);
              mma(st[2 * (i + j) + 1], term ? hi : lo, x[j][2], x[j][3]);
            }
      }
    }
    // the chunk's outputs as whole rows
#pragma unroll
    for (int i = 0; i < 8; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) stage_o[(i * 8 + t2 + (j & 1)) * SP + wid * 16 + g + (j >> 1) * 8] = pq[i][j];
    __syncthreads();
    const int t0 = chunk * CH, nt = min(CH, a.n - t0);
    constexpr int LANES = VT / 8;  // per row, eight columns each
#pragma unroll
    for (int i = tid; i < CH * LANES; i += THREADS) {
      const int t = i / LANES, c = (i - t * LANES) * 8;
      const float4 x = *reinterpret_cast<const float4 *>(stage_o + t * SP + c);
      const float4 y = *reinterpret_cast<const float4 *>(stage_o + t * SP + c + 4);
      const long long r = (long long)b * a.n + t0 + t;
      if (!s.normed) {
        if (t < nt && c < cols) {
          float *o = s.o + (r * a.heads + h) * a.vdim + vt + c;
          *reinterpret_cast<float4 *>(o) = x;
          *reinterpret_cast<float4 *>(o + 4) = y;
        }
        continue;
      }
      float q = x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w + y.x * y.x + y.y * y.y + y.z * y.z + y.w * y.w;
#pragma unroll
      for (int o = LANES / 2; o > 0; o >>= 1) q += __shfl_xor_sync(0xffffffffu, q, o);
      if (t >= nt || c >= cols) continue;
      const float inv = 1.0f / sqrtf(q / s.count + s.eps);
      const uint4 z = *reinterpret_cast<const uint4 *>(s.gate + r * s.in_ld + h * a.vdim + c);
      const float4 w0 = *reinterpret_cast<const float4 *>(s.norm + c), w1 = *reinterpret_cast<const float4 *>(s.norm + c + 4);
      *reinterpret_cast<uint4 *>(s.out + r * s.out_ld + h * a.vdim + c) =
          make_uint4(pack(x.x * inv * w0.x * silu_f32(low_half(z.x)), x.y * inv * w0.y * silu_f32(high_half(z.x))),
                     pack(x.z * inv * w0.z * silu_f32(low_half(z.y)), x.w * inv * w0.w * silu_f32(high_half(z.y))),
                     pack(y.x * inv * w1.x * silu_f32(low_half(z.z)), y.y * inv * w1.y * silu_f32(high_half(z.z))),
                     pack(y.z * inv * w1.z * silu_f32(low_half(z.w)), y.w * inv * w1.w * silu_f32(high_half(z.w))));
    }
    if (s.stages == 1 && chunk + 1 < a.chunks) load(chunk + 1);  // every warp is past this chunk's tiles
  }
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int d = i * 8 + t2 + (j & 1), v = v0 + (j >> 1) * 8;
      if (d < a.dim && v < a.vdim) S[(long long)d * a.vdim + v] = st[i][j];
    }
}

struct Parts {
  size_t mats, factors;
};
Parts parts(const DeltaMixer &m, long long rows, int streams) {
  const size_t all = (size_t)(rows / CH + streams) * m.heads;  // however the rows are shared among the streams
  return {all * 4 * MAT * 2, all * CH * 16};
}

constexpr size_t SMEM_LIMIT = 227 * 1024;

}  // namespace

bool delta_chunk_supports(const DeltaMixer &m) { return m.dim <= 256; }

size_t delta_chunk_bytes(const DeltaMixer &m, long long rows, int streams) {
  const Parts p = parts(m, rows, streams);
  return p.mats + p.factors;
}

int launch_delta_chunks(const DeltaMixer &m, const void *conv, float *o, void *scratch, const RowBatch &b, bool *normed,
                        cudaStream_t st, DevErr *err) {
  const Parts part = parts(m, b.rows(), b.streams);
  DeltaChunks c{};
  c.heads = m.heads;
  c.groups = m.groups;
  c.dim = m.dim;
  c.vdim = m.vdim;
  c.channels = m.conv_channels();
  c.n = b.n;
  c.chunks = (b.n + CH - 1) / CH;
  c.conv = static_cast<const bf16 *>(conv);
  c.mats = static_cast<bf16 *>(scratch);
  c.factors = reinterpret_cast<float *>(static_cast<char *>(scratch) + part.mats);
  const PrepareArgs p{c, 1.0f / sqrtf((float)m.true_dim), m.a_log, m.dt_bias, m.ba, m.ba_ld};
  const size_t vectors = (size_t)2 * CH * (m.dim + 8) * 2, floats = (size_t)2 * CH * TP * 4;
  const size_t prep_smem = vectors > floats ? vectors : floats;
  LB_CUDA(cudaFuncSetAttribute(delta_prepare_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)prep_smem));
  launch_pdl(delta_prepare_kernel, dim3((unsigned)c.chunks, (unsigned)m.heads, (unsigned)b.streams), dim3(PREP_THREADS),
             prep_smem, st, g_pdl_enabled, p);
  if (delta_scan_tc_supports(m)) {
    *normed = launch_delta_scan_tc(m, c, o, b, st, err);
    return 2;
  }
  ScanArgs s{};
  s.c = c;
  s.p0 = b.p0;
  s.slot0 = b.slot0;
  s.state = m.state;
  s.o = o;
  s.gate = static_cast<const bf16 *>(m.in) + c.channels;
  s.in_ld = m.in_ld;
  s.out_ld = m.out_ld;
  s.count = (float)m.true_vdim;
  s.eps = m.eps;
  s.norm = m.norm;
  s.out = static_cast<bf16 *>(m.out);
  // the widest tile of value columns that still gives about half the SMs a CTA
  const long long lanes = (long long)b.streams * m.heads;
  int vt = m.dim > 128 ? 64 : 128;
  while (vt > 32 && (vt / 2 >= m.vdim || lanes * ((m.vdim + vt - 1) / vt) < 74)) vt /= 2;
  s.normed = vt >= m.vdim;
  *normed = s.normed != 0;
  auto scan = [&](auto kernel, int warps) {
    const size_t stage = (size_t)stage_elems(m.dim, vt) * 2, extra = (size_t)CH * (vt + 4) * 4;
    s.stages = 2 * stage + extra <= SMEM_LIMIT ? 2 : 1;
    const size_t smem = s.stages * stage + extra;
    LB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    launch_pdl(kernel, dim3((unsigned)(m.heads * ((m.vdim + vt - 1) / vt)), (unsigned)b.streams), dim3((unsigned)(warps * 32)),
               smem, st, g_pdl_enabled, s);
  };
  if (m.dim <= 64) {
    if (vt == 128) scan(delta_scan_kernel<8, 8, false>, 8);
    else if (vt == 64) scan(delta_scan_kernel<8, 4, false>, 4);
    else scan(delta_scan_kernel<8, 2, false>, 2);
  } else if (m.dim <= 128) {
    if (vt == 128) scan(delta_scan_kernel<16, 8, false>, 8);
    else if (vt == 64) scan(delta_scan_kernel<16, 4, false>, 4);
    else scan(delta_scan_kernel<16, 2, false>, 2);
  } else {
    if (vt == 64) scan(delta_scan_kernel<32, 4, true>, 4);
    else scan(delta_scan_kernel<32, 2, true>, 2);
  }
  return 2;
}

}  // namespace lb
