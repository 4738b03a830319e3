// Sliding-window attention over a cache of latents: one compressed row c_j per position, from which
// head h's key is (W_uk c_j)_h and its value (W_uv c_j)_h, both linear, no positions in the scores.
//
//   s_ij = scale * q_i . k_j     for 0 <= i - j < window,   p = softmax_j(s),   o_i = sum_j p_ij v_j
//
// Because keys are linear in c, q . (W_uk c) = (W_uk^T q) . c: the kernels here take the product with
// W_uk to the query's side and the one with W_uv behind the weighted sum, so a step reads the window's
// latents once for all heads and expands no key or value.
//
//   latent_store_kernel          RMS norm of the new rows' W_dkv h into the cache, and the window's rows
//                                side by side for the expanding kernels (prefill_attention_tc.cu)
//   latent_attention_rows_kernel any size, one CTA per row and head, float or bfloat16 storage
//   latent_query / latent_chunk / latent_join   few rows on bfloat16: the absorbed query per head (and the
//                                new latents into the cache, by CTAs of their own); splits of the window
//                                for 16 heads at a time on mma.sync tiles, the 32-bit query and weights
//                                entering as two bfloat16 terms each; the join of the splits and W_uv,
//                                inside the same launch where the splits fit a thread-block cluster
// Scores, weights and norms are 32-bit throughout.
#include "model.cuh"
#include "tc_ptx.cuh"

#include <cuda_bf16.h>

namespace lb {

namespace {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float *p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16 *p, float v) { *p = __float2bfloat16_rn(v); }

__device__ __forceinline__ void put4(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
__device__ __forceinline__ void put4(bf16 *p, float4 v) {
  const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
  uint2 u;
  u.x = *reinterpret_cast<const unsigned *>(&a);
  u.y = *reinterpret_cast<const unsigned *>(&b);
  *reinterpret_cast<uint2 *>(p) = u;
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
  return v;
}

// ---- latents -------------------------------------------------------------------

// The latent of one new position by one warp: RMS norm of its W_dkv h row, zeros behind the rank.
template <typename T>
__device__ __forceinline__ void store_latent(const float *src, const float *__restrict__ gain, float eps, int rank,
                                             int ld, T *row, T *copy, int lane) {
  float s = 0.f;
  if ((rank & 3) == 0 && rank <= 1024) {  // the row in registers, four columns per lane and piece
    float4 v[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int c = (i * 32 + lane) * 4;
      v[i] = c < rank ? *reinterpret_cast<const float4 *>(src + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      s += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
    }
    const float inv = 1.0f / sqrtf(warp_sum(s) / (float)rank + eps);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
      const int c = (i * 32 + lane) * 4;
      if (c >= ld) break;
      const float4 g = c < rank ? *reinterpret_cast<const float4 *>(gain + c) : make_float4(0.f, 0.f, 0.f, 0.f);
      const float4 o = make_float4(v[i].x * inv * g.x, v[i].y * inv * g.y, v[i].z * inv * g.z, v[i].w * inv * g.w);
      put4(row + c, o);
      if (copy) put4(copy + c, o);
    }
    return;
  }
  for (int c = lane; c < rank; c += 32) s = fmaf(src[c], src[c], s);
  const float inv = 1.0f / sqrtf(warp_sum(s) / (float)rank + eps);
  for (int c = lane; c < ld; c += 32) {
    const float v = c < rank ? src[c] * inv * gain[c] : 0.f;
    put(row + c, v);
    if (copy) put(copy + c, v);
  }
}

// One warp per position: positions first .. p0 + n - 1 (first <= p0) of stream b. Old positions are
// copied from the cache to the packed rows, new ones normalised (dkv given) or, for a layer that uses
// another layer's latents, copied as well.
template <typename T>
__global__ void __launch_bounds__(256)
latent_store_kernel(const float *dkv, int dkv_ld, const float *__restrict__ gain, float eps, T *cache,
                    int cap, int ld, int rank, T *packed, int packed_rows, int first, int n, int p0_host,
                    const LoopState *state, int slot0) {
  pdl_launch_dependents();
  pdl_wait();
  const int b = blockIdx.y, lane = threadIdx.x & 31;
  const int p0 = state ? state->s - n : p0_host;
  const int from = packed ? first : p0;
  const int p = from + blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
  if (p >= p0 + n) return;
  T *row = cache + ((long long)(slot0 + b) * cap + p) * ld;
  T *dst = packed ? packed + ((long long)b * packed_rows + (p - first)) * ld : nullptr;
  if (p < p0 || dkv == nullptr) {
    if (dst == nullptr) return;
    const uint4 *src4 = reinterpret_cast<const uint4 *>(row);
    uint4 *dst4 = reinterpret_cast<uint4 *>(dst);
    for (int c = lane; c < ld * (int)sizeof(T) / 16; c += 32) dst4[c] = src4[c];
    return;
  }
  store_latent(dkv + ((long long)b * n + (p - p0)) * dkv_ld, gain, eps, rank, ld, row, dst, lane);
}

// ---- any size ------------------------------------------------------------------

constexpr int LR_THREADS = 256;
constexpr int LR_KEYS = 64;  // keys per pass

template <typename T>
__global__ void __launch_bounds__(LR_THREADS)
latent_attention_rows_kernel(const T *q, int q_ld, const T *__restrict__ w_uk, const T *__restrict__ w_uv,
                             int w_ld, const T *cache, int cap, int ld, int rank, int dim, int vdim, float scale,
                             int window, T *out, int out_ld, int n, int p0_host, const LoopState *state,
                             int slot0) {
  extern __shared__ float sm[];
  float *qa = sm;              // [rank] absorbed, scaled query
  float *acc = qa + rank;      // [rank] sum of weights times latents
  float *sc = acc + rank;      // [LR_KEYS] scores, then weights
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.y, lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  const int b = blockIdx.x / n, t = blockIdx.x - b * n;
  const long long r = blockIdx.x;
  const int p = (state ? state->s - n : p0_host) + t;
  const int lo = max(0, p - window + 1);
  const T *rows = cache + (long long)(slot0 + b) * cap * ld;
  const T *qr = q + r * q_ld + (long long)h * dim;
  for (int c = threadIdx.x; c < rank; c += LR_THREADS) {
    float s = 0.f;
    for (int e = 0; e < dim; ++e) s = fmaf(to_f(qr[e]), to_f(w_uk[((long long)h * dim + e) * w_ld + c]), s);
    qa[c] = s * scale;
    acc[c] = 0.f;
  }
  __syncthreads();
  float m = -INFINITY, l = 0.f;  // the same in every thread
  for (int j0 = lo; j0 <= p; j0 += LR_KEYS) {
    const int nk = min(LR_KEYS, p - j0 + 1);
    for (int j = wid; j < nk; j += LR_THREADS / 32) {
      const T *c = rows + (long long)(j0 + j) * ld;
      float s = 0.f;
      for (int i = lane; i < rank; i += 32) s = fmaf(qa[i], to_f(c[i]), s);
      s = warp_sum(s);
      if (lane == 0) sc[j] = s;
    }
    __syncthreads();
    float mt = -INFINITY;
    for (int j = lane; j < nk; j += 32) mt = fmaxf(mt, sc[j]);
    const float m_new = fmaxf(m, warp_max(mt));
    const float keep = expf(m - m_new);  // 0 on the first pass
    __syncthreads();
    for (int j = threadIdx.x; j < nk; j += LR_THREADS) sc[j] = expf(sc[j] - m_new);
    __syncthreads();
    float ls = 0.f;
    for (int j = lane; j < nk; j += 32) ls += sc[j];
    l = l * keep + warp_sum(ls);
    m = m_new;
    for (int c = threadIdx.x; c < rank; c += LR_THREADS) {
      float a = acc[c] * keep;
      for (int j = 0; j < nk; ++j) a = fmaf(sc[j], to_f(rows[(long long)(j0 + j) * ld + c]), a);
      acc[c] = a;
    }
    __syncthreads();
  }
  const float inv = 1.0f / l;
  for (int e = wid; e < vdim; e += LR_THREADS / 32) {
    const T *wr = w_uv + ((long long)h * vdim + e) * w_ld;
    float s = 0.f;
    for (int i = lane; i < rank; i += 32) s = fmaf(to_f(wr[i]), acc[i], s);
    s = warp_sum(s);
    if (lane == 0) put(out + r * out_ld + (long long)h * vdim + e, s * inv);
  }
}

// ---- few rows on bfloat16 --------------------------------------------------------

constexpr int LD_KEYS = 64;      // keys per tile
constexpr int LD_HEADS = 16;     // heads per CTA: the rows of an mma tile
constexpr int LD_THREADS = 256;
constexpr int LQ_COLS = 256;     // latent columns per CTA of the query kernel, eight per thread
constexpr int LD_ROWS = 4;       // rows per CTA of the query and join kernels
constexpr int LD_CLUSTER = 8;    // CTAs of the largest cluster
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ void mma_bf16(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
      : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldmatrix_x2_trans(unsigned &r0, unsigned &r1, const void *p) {
  const unsigned addr = (unsigned)__cvta_generic_to_shared(p);
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.trans.shared.b16 {%0, %1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
// 16 bytes to shared memory in the background; bytes = 0 stores zeros.
__device__ __forceinline__ void copy16(void *dst, const void *src, int bytes) {
  const unsigned addr = (unsigned)__cvta_generic_to_shared(dst);
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(addr), "l"(src), "r"(bytes) : "memory");
}
__device__ __forceinline__ void copy_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void copy_wait() {
  asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}
__device__ __forceinline__ void split2(float v, bf16 &hi, bf16 &lo) {
  hi = __float2bfloat16_rn(v);
  lo = __float2bfloat16_rn(v - __bfloat162float(hi));
}
__device__ __forceinline__ void unpack8(uint4 v, float (&f)[8]) {
  const unsigned u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    f[2 * i] = __uint_as_float(u[i] << 16);
    f[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u);
  }
}

// What the few-row kernels share. The absorbed queries are [rows][heads16][rk] in two bfloat16 terms
// (heads16: heads rounded up to 16, rk: rank rounded up to 16), the partial results [rows][heads][splits].
struct LdShape {
  int heads, heads16, dim, vdim, rank, rk, rank4, window, splits, span;  // span: keys per split, a multiple of LD_KEYS
  int n, p0, slot0;
  const LoopState *state;
  __device__ int position(long long r, int &b) const {
    b = (int)(r / n);
    return (state ? state->s - n : p0) + (int)(r - (long long)b * n);
  }
};

// (hi + lo)[r, h, c] = scale * log2(e) * sum_e q[r, h, e] W_uk[h, e, c] for ROWS rows of one head; the
// eight warps take every eighth e. CTAs behind the last head (a layer with latents of its own) put the new
// rows' latents into the cache meanwhile.
template <int ROWS>
__global__ void __launch_bounds__(LD_THREADS)
latent_query_kernel(LdShape g, const bf16 *q, int q_ld, const bf16 *__restrict__ w_uk, int w_ld, float factor,
                    long long n_rows, bf16 *qh, bf16 *ql, LatentFresh fresh,
                    bf16 *cache, int cap, int ld) {
  __shared__ __align__(16) float part[8][ROWS][LQ_COLS];
  extern __shared__ float qs[];  // [ROWS][dim]
  pdl_launch_dependents();
  const int h = blockIdx.y, lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  const int c = blockIdx.x * LQ_COLS + lane * 8;
  constexpr int PRE = 4;  // rows of W_uk per warp that are requested ahead of the wait
  uint4 pre[PRE];
  const bf16 *w = w_uk + (long long)h * g.dim * w_ld + c;  // rows end on a multiple of 8 with zeros behind the rank
#pragma unroll
  for (int i = 0; i < PRE; ++i)
    pre[i] = h < g.heads && c < g.rank && wid + 8 * i < g.dim
                 ? *reinterpret_cast<const uint4 *>(w + (long long)(wid + 8 * i) * w_ld)
                 : make_uint4(0, 0, 0, 0);
  pdl_wait();
  const long long r0 = (long long)blockIdx.z * ROWS;
  const int nr = (int)min((long long)ROWS, n_rows - r0);
  if (h == g.heads) {
    if (blockIdx.x == 0 && wid < nr) {
      int b;
      const int p = g.position(r0 + wid, b);
      store_latent(fresh.dkv + (r0 + wid) * fresh.ld, fresh.gain, fresh.eps, g.rank, ld,
                   cache + ((long long)(g.slot0 + b) * cap + p) * ld, (bf16 *)nullptr, lane);
    }
    return;
  }
  for (int i = threadIdx.x; i < ROWS * g.dim; i += LD_THREADS) {
    const int r = i / g.dim, e = i - r * g.dim;
    qs[i] = r < nr ? to_f(q[(r0 + r) * q_ld + (long long)h * g.dim + e]) : 0.f;
  }
  float acc[ROWS][8] = {};
  __syncthreads();
  auto add = [&](int e, uint4 row) {
    float f[8];
    unpack8(row, f);
#pragma unroll
    for (int r = 0; r < ROWS; ++r) {
      const float v = qs[r * g.dim + e];
#pragma unroll
      for (int k = 0; k < 8; ++k) acc[r][k] = fmaf(v, f[k], acc[r][k]);
    }
  };
  if (c < g.rank) {
#pragma unroll
    for (int i = 0; i < PRE; ++i)
      if (wid + 8 * i < g.dim) add(wid + 8 * i, pre[i]);
#pragma unroll 4
    for (int e = wid + 8 * PRE; e < g.dim; e += 8) add(e, *reinterpret_cast<const uint4 *>(w + (long long)e * w_ld));
  }
#pragma unroll
  for (int r = 0; r < ROWS; ++r) {
    *reinterpret_cast<float4 *>(&part[wid][r][lane * 8]) = make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]);
    *reinterpret_cast<float4 *>(&part[wid][r][lane * 8 + 4]) = make_float4(acc[r][4], acc[r][5], acc[r][6], acc[r][7]);
  }
  __syncthreads();
  const int col = blockIdx.x * LQ_COLS + threadIdx.x;
  if (col >= g.rk) return;
  for (int r = 0; r < nr; ++r) {
    float v = 0.f;
#pragma unroll
    for (int k = 0; k < 8; ++k) v += part[k][r][threadIdx.x];
    const long long at = ((r0 + r) * g.heads16 + h) * g.rk + col;
    bf16 hi, lo;
    split2(col < g.rank ? v * factor : 0.f, hi, lo);
    qh[at] = hi;
    ql[at] = lo;
  }
}

// Split blockIdx.x (span keys from the window's first one on) of row blockIdx.z for 16 heads: tiles of 64
// keys, the next one's latents on their way while a tile is used (stages == 2), running maximum and
// sum per head, o[head][rank] = sum_j 2^(s_j - m) c_j in registers. NT: tiles of 8 latent columns per warp.
// CLUSTER: the splits of a row and head group are the CTAs of a thread-block cluster; their results meet in
// shared memory, each CTA joins its share of the heads and maps it through W_uv (latent_join_kernel does
// both where the splits are too many for a cluster).
template <int NT, bool CLUSTER>
__global__ void __launch_bounds__(LD_THREADS)
latent_chunk_kernel(LdShape g, const bf16 *q_hi, const bf16 *q_lo, const bf16 *cache,
                    int cap, int ld, int stages, float *part_o, float2 *part_ml, const bf16 *__restrict__ w_uv, int w_ld,
                    bf16 *out, int out_ld) {
  extern __shared__ __align__(16) unsigned char smraw[];
  const int rk = g.rk, pitch = rk + 8;               // 16-byte rows whose fragments hit distinct banks
  bf16 *qh = reinterpret_cast<bf16 *>(smraw);        // [16][pitch] high and low terms of the query
  bf16 *ql = qh + LD_HEADS * pitch;
  constexpr int PP = LD_KEYS + 8, SP = LD_KEYS + 4;
  bf16 *ph = ql + LD_HEADS * pitch;                  // [16][PP] high and low terms of the weights
  bf16 *pl = ph + LD_HEADS * PP;
  float *sc = reinterpret_cast<float *>(pl + LD_HEADS * PP);  // [16][SP]
  float *fac = sc + LD_HEADS * SP;                   // [16] factors of what has been summed so far
  bf16 *tiles = reinterpret_cast<bf16 *>(fac + LD_HEADS);     // [stages][LD_KEYS][pitch]
  pdl_launch_dependents();
  if constexpr (CLUSTER) {  // the value rows this CTA maps its heads through depend on nothing: towards L2 now
    const int nh = min(LD_HEADS, g.heads - (int)blockIdx.y * LD_HEADS);
    for (int hh = blockIdx.x; hh < nh; hh += g.splits) {
      const char *rows = reinterpret_cast<const char *>(w_uv + (long long)(blockIdx.y * LD_HEADS + hh) * g.vdim * w_ld);
      for (int at = threadIdx.x * 128; at < g.vdim * w_ld * 2; at += LD_THREADS * 128)
        asm volatile("prefetch.global.L2 [%0];" ::"l"(rows + at));
    }
  }
  pdl_wait();
  const long long r = blockIdx.z;
  int b;
  const int p = g.position(r, b);
  const int j0 = max(0, p - g.window + 1) + blockIdx.x * g.span;
  if (!CLUSTER && j0 > p) return;
  const int total = max(0, min(g.span, p - j0 + 1)), nt = (total + LD_KEYS - 1) / LD_KEYS;
  const int h0 = blockIdx.y * LD_HEADS, nh = min(LD_HEADS, g.heads - h0);
  const int tid = threadIdx.x, lane = tid & 31, wid = tid >> 5;
  const int gr = lane >> 2, tq = lane & 3;
  const bf16 *src = cache + ((long long)(g.slot0 + b) * cap + j0) * ld;
  const int pieces = rk >> 3;
  auto fetch = [&](int tile) {  // the cache's rows end on a multiple of 8 columns with zeros behind the rank
    bf16 *dst = tiles + (tile % stages) * LD_KEYS * pitch;
    const int k0 = tile * LD_KEYS;
#pragma unroll 4
    for (int i = tid; i < LD_KEYS * pieces; i += LD_THREADS) {
      const int j = i / pieces, c = (i - j * pieces) * 8;
      const bool in = k0 + j < total && c < ld;
      copy16(dst + j * pitch + c, in ? src + (long long)(k0 + j) * ld + c : src, in ? 16 : 0);
    }
    copy_commit();
  };
  {
    const long long at = (r * g.heads16 + h0) * rk;
#pragma unroll 4
    for (int i = tid; i < LD_HEADS * pieces; i += LD_THREADS) {
      const int hh = i / pieces, c = (i - hh * pieces) * 8;
      copy16(qh + hh * pitch + c, q_hi + at + hh * rk + c, 16);
      copy16(ql + hh * pitch + c, q_lo + at + hh * rk + c, 16);
    }
  }
  if (nt > 0) fetch(0);
  else copy_commit();
  float o[NT][4];
#pragma unroll
  for (int i = 0; i < NT; ++i)
#pragma unroll
    for (int k = 0; k < 4; ++k) o[i][k] = 0.f;
  float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};  // of heads 2 * wid and 2 * wid + 1, in every lane
  for (int tile = 0; tile < nt; ++tile) {
    if (stages > 1 && tile + 1 < nt) {
      fetch(tile + 1);
      copy_wait<1>();
    } else {
      copy_wait<0>();
    }
    __syncthreads();
    const bf16 *ck = tiles + (tile % stages) * LD_KEYS * pitch;
    const int nk = min(LD_KEYS, total - tile * LD_KEYS);
    {  // scores: warp w takes keys 8w .. 8w + 7; two accumulators keep the products of the terms apart
      float d[4] = {0.f, 0.f, 0.f, 0.f}, d2[4] = {0.f, 0.f, 0.f, 0.f};
      const bf16 *kr = ck + (wid * 8 + gr) * pitch + tq * 2;
      const bf16 *ah = qh + gr * pitch + tq * 2, *al = ql + gr * pitch + tq * 2;
#pragma unroll 4
      for (int k = 0; k < rk; k += 16) {
        const unsigned b0 = *reinterpret_cast<const unsigned *>(kr + k), b1 = *reinterpret_cast<const unsigned *>(kr + k + 8);
        const unsigned a[4] = {*reinterpret_cast<const unsigned *>(ah + k),
                               *reinterpret_cast<const unsigned *>(ah + k + 8 * pitch),
                               *reinterpret_cast<const unsigned *>(ah + k + 8),
                               *reinterpret_cast<const unsigned *>(ah + k + 8 * pitch + 8)};
        const unsigned a2[4] = {*reinterpret_cast<const unsigned *>(al + k),
                                *reinterpret_cast<const unsigned *>(al + k + 8 * pitch),
                                *reinterpret_cast<const unsigned *>(al + k + 8),
                                *reinterpret_cast<const unsigned *>(al + k + 8 * pitch + 8)};
        mma_bf16(d2, a2, b0, b1);
        mma_bf16(d, a, b0, b1);
      }
      const int j = wid * 8 + tq * 2;
      *reinterpret_cast<float2 *>(sc + gr * SP + j) = make_float2(d[0] + d2[0], d[1] + d2[1]);
      *reinterpret_cast<float2 *>(sc + (gr + 8) * SP + j) = make_float2(d[2] + d2[2], d[3] + d2[3]);
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 2; ++i) {  // weights: a lane takes two keys
      const int hh = wid * 2 + i;
      const float s0 = lane < nk ? sc[hh * SP + lane] : -INFINITY;
      const float s1 = lane + 32 < nk ? sc[hh * SP + lane + 32] : -INFINITY;
      const float mn = fmaxf(m[i], warp_max(fmaxf(s0, s1)));
      const float p0 = exp2f(s0 - mn), p1 = exp2f(s1 - mn), keep = exp2f(m[i] - mn);
      l[i] = l[i] * keep + warp_sum(p0 + p1);
      m[i] = mn;
      bf16 hi, low;
      split2(p0, hi, low);
      ph[hh * PP + lane] = hi;
      pl[hh * PP + lane] = low;
      split2(p1, hi, low);
      ph[hh * PP + lane + 32] = hi;
      pl[hh * PP + lane + 32] = low;
      if (lane == 0) fac[hh] = keep;
    }
    __syncthreads();
    unsigned a[LD_KEYS / 16][4], a2[LD_KEYS / 16][4];
#pragma unroll
    for (int k = 0; k < LD_KEYS / 16; ++k) {
      const bf16 *x = ph + gr * PP + tq * 2 + k * 16, *y = pl + gr * PP + tq * 2 + k * 16;
      a[k][0] = *reinterpret_cast<const unsigned *>(x);
      a[k][1] = *reinterpret_cast<const unsigned *>(x + 8 * PP);
      a[k][2] = *reinterpret_cast<const unsigned *>(x + 8);
      a[k][3] = *reinterpret_cast<const unsigned *>(x + 8 * PP + 8);
      a2[k][0] = *reinterpret_cast<const unsigned *>(y);
      a2[k][1] = *reinterpret_cast<const unsigned *>(y + 8 * PP);
      a2[k][2] = *reinterpret_cast<const unsigned *>(y + 8);
      a2[k][3] = *reinterpret_cast<const unsigned *>(y + 8 * PP + 8);
    }
    const float f0 = fac[gr], f1 = fac[gr + 8];
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int c0 = (i * 8 + wid) * 8;
      if (c0 < rk) {
        o[i][0] *= f0;
        o[i][1] *= f0;
        o[i][2] *= f1;
        o[i][3] *= f1;
#pragma unroll
        for (int k = 0; k < LD_KEYS / 16; ++k) {
          unsigned b0, b1;
          ldmatrix_x2_trans(b0, b1, ck + (k * 16 + (lane & 15)) * pitch + c0);
          mma_bf16(o[i], a2[k], b0, b1);
          mma_bf16(o[i], a[k], b0, b1);
        }
      }
    }
    if (stages == 1 && tile + 1 < nt) {
      __syncthreads();
      fetch(tile + 1);
    } else if (stages > 1) {
      __syncthreads();  // the tile after next goes over this one
    }
  }
  if constexpr (CLUSTER) {
    copy_wait<0>();
    __syncthreads();  // the tiles' space becomes this split's results: [16][rank4], then [16] (maximum, sum)
    float *os = reinterpret_cast<float *>(tiles);
    float2 *mls = reinterpret_cast<float2 *>(os + LD_HEADS * g.rank4);
    const int r8 = (g.rank + 7) & ~7, ranks = g.splits;
    const int share = (nh - (int)blockIdx.x + ranks - 1) / ranks;  // heads blockIdx.x, blockIdx.x + ranks, ... are this CTA's
    float *ol = reinterpret_cast<float *>(qh);                     // [share][r8] weighted latents, over the queries
    float *join = sc;                                              // [share][8] factors of the splits, over the scores
#pragma unroll
    for (int i = 0; i < 2; ++i)
      if (lane == 0) mls[wid * 2 + i] = make_float2(m[i], l[i]);
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int c = (i * 8 + wid) * 8 + tq * 2;
      if (c >= g.rank4) continue;
      *reinterpret_cast<float2 *>(os + gr * g.rank4 + c) = make_float2(o[i][0], o[i][1]);
      *reinterpret_cast<float2 *>(os + (gr + 8) * g.rank4 + c) = make_float2(o[i][2], o[i][3]);
    }
    __syncwarp();
    cluster_sync_all();
    const unsigned os_at = smem_u32(os), ml_at = smem_u32(mls);
    for (int i = wid; i < share; i += LD_THREADS / 32) {  // lane q looks at split q
      const unsigned at = ml_at + (unsigned)((int)blockIdx.x + i * ranks) * 8u;
      const float mq = lane < ranks ? ld_cluster_f32(cluster_map(at, (unsigned)lane)) : -INFINITY;
      const float lq = lane < ranks ? ld_cluster_f32(cluster_map(at + 4u, (unsigned)lane)) : 0.f;
      const float e = exp2f(mq - warp_max(mq));
      const float sum = warp_sum(lq * e);
      if (lane < ranks) join[i * LD_CLUSTER + lane] = e / sum;
    }
    __syncthreads();
    const int cols = r8 >> 2;
    for (int k = tid; k < share * cols; k += LD_THREADS) {
      const int i = k / cols, c = (k - i * cols) * 4;
      float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < g.rank4) {
        const unsigned at = os_at + (unsigned)(((int)blockIdx.x + i * ranks) * g.rank4 + c) * 4u;
        float4 v[LD_CLUSTER];
#pragma unroll
        for (int q = 0; q < LD_CLUSTER; ++q)
          v[q] = q < ranks ? ld_cluster_f4(cluster_map(at, (unsigned)q)) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int q = 0; q < LD_CLUSTER; ++q)
          if (q < ranks) {
            const float f = join[i * LD_CLUSTER + q];
            acc = make_float4(fmaf(f, v[q].x, acc.x), fmaf(f, v[q].y, acc.y), fmaf(f, v[q].z, acc.z), fmaf(f, v[q].w, acc.w));
          }
      }
      *reinterpret_cast<float4 *>(ol + i * r8 + c) = acc;
    }
    __syncthreads();
    // the value rows of all the CTA's heads, four per warp and trip; a row's loads precede their use
    const int n_rows = share * g.vdim;
    for (int k0 = wid * 4; k0 < n_rows; k0 += LD_THREADS / 32 * 4) {
      float sum[4] = {};
      const bf16 *wr[4];
      const float *x[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int k = min(k0 + u, n_rows - 1), i = k / g.vdim, e = k - i * g.vdim;
        wr[u] = w_uv + ((long long)(h0 + (int)blockIdx.x + i * ranks) * g.vdim + e) * w_ld;
        x[u] = ol + i * r8;
      }
      for (int c = lane * 8; c < r8; c += 256) {
        uint4 w4[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) w4[u] = *reinterpret_cast<const uint4 *>(wr[u] + c);
#pragma unroll
        for (int u = 0; u < 4; ++u) {
          float f[8];
          unpack8(w4[u], f);
          const float4 y = *reinterpret_cast<const float4 *>(x[u] + c), z = *reinterpret_cast<const float4 *>(x[u] + c + 4);
          sum[u] = fmaf(f[0], y.x, fmaf(f[1], y.y, fmaf(f[2], y.z, fmaf(f[3], y.w, sum[u]))));
          sum[u] = fmaf(f[4], z.x, fmaf(f[5], z.y, fmaf(f[6], z.z, fmaf(f[7], z.w, sum[u]))));
        }
      }
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const float v = warp_sum(sum[u]);
        const int k = k0 + u, i = k / g.vdim;
        if (lane == 0 && k < n_rows)
          out[r * out_ld + (long long)(h0 + (int)blockIdx.x + i * ranks) * g.vdim + (k - i * g.vdim)] = __float2bfloat16_rn(v);
      }
    }
    __syncwarp();
    cluster_sync_all();  // a split's shared memory stays until every other has read it
  } else {
#pragma unroll
    for (int i = 0; i < 2; ++i)
      if (lane == 0 && wid * 2 + i < nh)
        part_ml[(r * g.heads + h0 + wid * 2 + i) * g.splits + blockIdx.x] = make_float2(m[i], l[i]);
#pragma unroll
    for (int i = 0; i < NT; ++i) {
      const int c = (i * 8 + wid) * 8 + tq * 2;
      if (c >= g.rank4) continue;  // columns behind the rank are zeros
#pragma unroll
      for (int k = 0; k < 2; ++k)
        if (gr + 8 * k < nh)
          *reinterpret_cast<float2 *>(part_o + ((r * g.heads + h0 + gr + 8 * k) * g.splits + blockIdx.x) * (long long)g.rank4 +
                                      c) = make_float2(o[i][2 * k], o[i][2 * k + 1]);
    }
  }
}

// Joins the splits of LD_ROWS rows of one head and maps the weighted latents through W_uv; the CTAs of
// grid.y share the head's value rows.
// PIECES: pieces of 256 latent columns a row of W_uv has (at most).
template <int PIECES>
__global__ void __launch_bounds__(LD_THREADS)
latent_join_kernel(LdShape g, const float *part_o, const float2 *part_ml, const bf16 *__restrict__ w_uv,
                   int w_ld, long long n_rows, bf16 *out, int out_ld) {
  extern __shared__ __align__(16) float ol[];  // [LD_ROWS][rank rounded up to 8] weighted latents, then [LD_ROWS][splits]
  pdl_launch_dependents();
  const int h = blockIdx.x, lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  const long long r0 = (long long)blockIdx.z * LD_ROWS;
  const int nr = (int)min((long long)LD_ROWS, n_rows - r0);
  const int r8 = (g.rank + 7) & ~7;
  const int e_per = (g.vdim + gridDim.y - 1) / gridDim.y;
  const int e0 = blockIdx.y * e_per + wid, e1 = min(g.vdim, (int)(blockIdx.y + 1) * e_per);
  constexpr int PRE = 4 / PIECES;  // value rows per warp that are requested ahead of the wait
  const bf16 *wv = w_uv + (long long)h * g.vdim * w_ld;  // rows end on a multiple of 8 with zeros behind the rank
  auto piece = [&](int e, int i) {
    const int c = (i * 32 + lane) * 8;
    return e < e1 && c < r8 ? *reinterpret_cast<const uint4 *>(wv + (long long)e * w_ld + c) : make_uint4(0, 0, 0, 0);
  };
  uint4 pre[PRE][PIECES];
#pragma unroll
  for (int k = 0; k < PRE; ++k)
#pragma unroll
    for (int i = 0; i < PIECES; ++i) pre[k][i] = piece(e0 + 8 * k, i);
  pdl_wait();
  float *fac = ol + LD_ROWS * r8;
  __shared__ int counts[LD_ROWS];
  if (wid < nr) {
    int b;
    const int p = g.position(r0 + wid, b);
    const int nc = (min(g.window, p + 1) + g.span - 1) / g.span;
    const float2 *ml = part_ml + ((r0 + wid) * g.heads + h) * g.splits;
    float m = -INFINITY, l = 0.f;
    for (int c = lane; c < nc; c += 32) m = fmaxf(m, ml[c].x);
    m = warp_max(m);
    for (int c = lane; c < nc; c += 32) l += ml[c].y * exp2f(ml[c].x - m);
    l = warp_sum(l);
    for (int c = lane; c < nc; c += 32) fac[wid * g.splits + c] = exp2f(ml[c].x - m) / l;
    if (lane == 0) counts[wid] = nc;
  }
  __syncthreads();
  const int cols = r8 >> 2;
  for (int i = threadIdx.x; i < nr * cols; i += LD_THREADS) {
    const int r = i / cols, c = (i - r * cols) * 4;
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
    if (c < g.rank4) {
      const float *o = part_o + ((r0 + r) * g.heads + h) * (long long)g.splits * g.rank4 + c;
      const float *f = fac + r * g.splits;
      const int nc = counts[r];
#pragma unroll 4
      for (int k = 0; k < nc; ++k) {
        const float4 v = *reinterpret_cast<const float4 *>(o + (long long)k * g.rank4);
        a = make_float4(fmaf(f[k], v.x, a.x), fmaf(f[k], v.y, a.y), fmaf(f[k], v.z, a.z), fmaf(f[k], v.w, a.w));
      }
    }
    *reinterpret_cast<float4 *>(ol + r * r8 + c) = a;
  }
  __syncthreads();
  auto value = [&](int e, const uint4 (&row)[PIECES]) {
    float s[LD_ROWS] = {};
#pragma unroll
    for (int i = 0; i < PIECES; ++i) {
      const int c = (i * 32 + lane) * 8;
      if (c >= r8) break;
      float f[8];
      unpack8(row[i], f);
#pragma unroll
      for (int r = 0; r < LD_ROWS; ++r) {
        if (r >= nr) break;
        const float4 x = *reinterpret_cast<const float4 *>(ol + r * r8 + c), y = *reinterpret_cast<const float4 *>(ol + r * r8 + c + 4);
        s[r] = fmaf(f[0], x.x, fmaf(f[1], x.y, fmaf(f[2], x.z, fmaf(f[3], x.w, s[r]))));
        s[r] = fmaf(f[4], y.x, fmaf(f[5], y.y, fmaf(f[6], y.z, fmaf(f[7], y.w, s[r]))));
      }
    }
#pragma unroll
    for (int r = 0; r < LD_ROWS; ++r) {
      if (r >= nr) break;
      const float v = warp_sum(s[r]);
      if (lane == 0) out[(r0 + r) * out_ld + (long long)h * g.vdim + e] = __float2bfloat16_rn(v);
    }
  };
#pragma unroll
  for (int k = 0; k < PRE; ++k)
    if (e0 + 8 * k < e1) value(e0 + 8 * k, pre[k]);
  for (int e = e0 + 8 * PRE; e < e1; e += 8) {
    uint4 row[PIECES];
#pragma unroll
    for (int i = 0; i < PIECES; ++i) row[i] = piece(e, i);
    value(e, row);
  }
}

// (A cluster's join reuses the areas: the weighted latents, at most 16 rows of rank rounded up to 8 floats,
// over the queries, 32 rows of at least rank + 8 halves; a split's results, 16 rows of rank floats and 16
// pairs, over the first tile, 64 rows of at least rank + 8 halves.)
size_t chunk_smem(int rank, int stages) {
  const int pitch = ((rank + 15) & ~15) + 8;
  return (size_t)(stages * LD_KEYS + 2 * LD_HEADS) * pitch * 2 + (size_t)2 * LD_HEADS * (LD_KEYS + 8) * 2 +
         (size_t)LD_HEADS * (LD_KEYS + 4) * 4 + LD_HEADS * 4;
}
constexpr size_t LD_SMEM_LIMIT = 220 * 1024;

// How a window of `window` keys (contexts up to s_cap) is cut for so many rows: about two CTAs per SM.
int most_splits(int heads, int window, int s_cap, long long rows) {
  const int tiles = ((window < s_cap ? window : s_cap) + LD_KEYS - 1) / LD_KEYS;
  const long long groups = rows * ((heads + LD_HEADS - 1) / LD_HEADS);
  const long long want = (2 * 148 + groups - 1) / groups;
  return (int)(want < tiles ? want : tiles);
}
constexpr int LD_CLUSTER_TILES = 4;  // key tiles per CTA up to which a cluster beats more splits and a second launch
void plan_splits(int heads, int window, int s_cap, long long rows, int *splits, int *span) {
  const int tiles = ((window < s_cap ? window : s_cap) + LD_KEYS - 1) / LD_KEYS;
  int want = most_splits(heads, window, s_cap, rows);
  if (want > LD_CLUSTER && tiles <= LD_CLUSTER * LD_CLUSTER_TILES) want = LD_CLUSTER;
  const int per = (tiles + want - 1) / want;
  *span = per * LD_KEYS;
  *splits = (tiles + per - 1) / per;
}

struct LdScratch {
  size_t q, ml, o;  // floats: both query terms, maxima and sums, partial results
};
LdScratch ld_scratch(int heads, int rank, int splits, long long rows) {
  const size_t heads16 = (size_t)(heads + 15) / 16 * 16, rk = (size_t)(rank + 15) / 16 * 16;
  const size_t rh = (size_t)rows * heads;
  return {(size_t)rows * heads16 * rk, (rh * splits * 2 + 3) / 4 * 4, rh * splits * ((size_t)(rank + 3) / 4 * 4)};
}

}  // namespace

void launch_latent_store(const float *dkv, int dkv_ld, const float *gain, float eps, const LatentCache &cache,
                         void *packed, int packed_rows, int first, Precision type, const RowBatch &b, cudaStream_t st) {
  const int count = packed ? b.p0 + b.n - first : b.n;
  const dim3 grid((unsigned)((count + 7) / 8), (unsigned)b.streams);
  if (type == Precision::BF16)
    launch_pdl(latent_store_kernel<bf16>, grid, dim3(256), 0, st, g_pdl_enabled, dkv, dkv_ld, gain, eps,
               static_cast<bf16 *>(cache.rows), cache.cap, cache.ld, cache.rank, static_cast<bf16 *>(packed), packed_rows,
               first, b.n, b.p0, b.state, b.slot0);
  else
    launch_pdl(latent_store_kernel<float>, grid, dim3(256), 0, st, g_pdl_enabled, dkv, dkv_ld, gain, eps,
               static_cast<float *>(cache.rows), cache.cap, cache.ld, cache.rank, static_cast<float *>(packed), packed_rows,
               first, b.n, b.p0, b.state, b.slot0);
}

void launch_latent_attention_rows(const LatentAttention &a, Precision type, const RowBatch &b, cudaStream_t st) {
  const dim3 grid((unsigned)b.rows(), (unsigned)a.heads);
  const size_t smem = ((size_t)2 * a.cache.rank + LR_KEYS) * sizeof(float);
  auto go = [&](auto kernel, auto *tag) {
    using T = std::remove_pointer_t<decltype(tag)>;
    if (smem > 48 * 1024) LB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    launch_pdl(kernel, grid, dim3(LR_THREADS), smem, st, g_pdl_enabled, static_cast<const T *>(a.q), a.q_ld,
               static_cast<const T *>(a.w_uk), static_cast<const T *>(a.w_uv), a.w_ld,
               static_cast<const T *>(a.cache.rows), a.cache.cap, a.cache.ld, a.cache.rank, a.dim, a.vdim, a.scale, a.window,
               static_cast<T *>(a.out), a.out_ld, b.n, b.p0, b.state, b.slot0);
  };
  if (type == Precision::BF16) go(latent_attention_rows_kernel<bf16>, (bf16 *)nullptr);
  else go(latent_attention_rows_kernel<float>, (float *)nullptr);
}

bool latent_decode_supports(const LatentAttention &a) {
  return a.cache.rank <= 1024 && chunk_smem(a.cache.rank, 1) <= LD_SMEM_LIMIT && a.dim <= 2048;
}

size_t latent_decode_scratch_floats(int heads, int rank, int window, int s_cap, long long rows) {
  // fewer rows are cut into more splits, shorter contexts into no more than most_splits of the longest one
  size_t need = 0;
  for (long long r = 1; r <= rows; ++r) {
    const LdScratch n = ld_scratch(heads, rank, most_splits(heads, window, s_cap, r), r);
    need = n.q + n.ml + n.o > need ? n.q + n.ml + n.o : need;
  }
  return need;
}

int launch_latent_decode(const LatentAttention &a, const LatentFresh &fresh, float *scratch, const RowBatch &b,
                         cudaStream_t st) {
  const long long rows = b.rows();
  LdShape g{};
  g.heads = a.heads;
  g.heads16 = (a.heads + 15) / 16 * 16;
  g.dim = a.dim;
  g.vdim = a.vdim;
  g.rank = a.cache.rank;
  g.rk = (g.rank + 15) / 16 * 16;
  g.rank4 = (g.rank + 3) / 4 * 4;
  g.window = a.window;
  g.n = b.n;
  g.p0 = b.p0;
  g.slot0 = b.slot0;
  g.state = b.state;
  plan_splits(a.heads, a.window, b.s_cap, rows, &g.splits, &g.span);
  const LdScratch n = ld_scratch(a.heads, g.rank, g.splits, rows);
  bf16 *qh = reinterpret_cast<bf16 *>(scratch), *ql = qh + n.q;
  float2 *ml = reinterpret_cast<float2 *>(scratch + n.q);
  float *po = scratch + n.q + n.ml;
  const bf16 *cache = static_cast<const bf16 *>(a.cache.rows);
  const unsigned row_groups = (unsigned)((rows + LD_ROWS - 1) / LD_ROWS);
  auto query = [&](auto kernel, int per) {
    const size_t q_smem = (size_t)per * a.dim * sizeof(float);
    if (q_smem + (size_t)8 * per * LQ_COLS * 4 > 48 * 1024)
      LB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)q_smem));
    launch_pdl(kernel,
               dim3((unsigned)((g.rk + LQ_COLS - 1) / LQ_COLS), (unsigned)(a.heads + (fresh.dkv ? 1 : 0)),
                    (unsigned)((rows + per - 1) / per)),
               dim3(LD_THREADS), q_smem, st, g_pdl_enabled, g, static_cast<const bf16 *>(a.q), a.q_ld,
               static_cast<const bf16 *>(a.w_uk), a.w_ld, a.scale * LOG2E, rows, qh, ql, fresh,
               static_cast<bf16 *>(a.cache.rows), a.cache.cap, a.cache.ld);
  };
  if (rows < LD_ROWS) query(latent_query_kernel<1>, 1);
  else query(latent_query_kernel<LD_ROWS>, LD_ROWS);
  const int stages = g.span > LD_KEYS && chunk_smem(g.rank, 2) <= LD_SMEM_LIMIT ? 2 : 1;
  const size_t smem = chunk_smem(g.rank, stages);
  const bool cluster = g.splits <= LD_CLUSTER;
  auto chunk = [&](auto kernel) {
    if (smem > 48 * 1024) LB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    launch_pdl_cluster_x(kernel, dim3((unsigned)g.splits, (unsigned)(g.heads16 / LD_HEADS), (unsigned)rows), dim3(LD_THREADS),
                         smem, st, g_pdl_enabled, cluster ? (unsigned)g.splits : 1u, g, (const bf16 *)qh, (const bf16 *)ql,
                         cache, a.cache.cap, a.cache.ld, stages, po, ml, static_cast<const bf16 *>(a.w_uv), a.w_ld,
                         static_cast<bf16 *>(a.out), a.out_ld);
  };
  if (cluster) {
    if (g.rk <= 128) chunk(latent_chunk_kernel<2, true>);
    else if (g.rk <= 256) chunk(latent_chunk_kernel<4, true>);
    else if (g.rk <= 512) chunk(latent_chunk_kernel<8, true>);
    else chunk(latent_chunk_kernel<16, true>);
    return 2;
  }
  if (g.rk <= 128) chunk(latent_chunk_kernel<2, false>);
  else if (g.rk <= 256) chunk(latent_chunk_kernel<4, false>);
  else if (g.rk <= 512) chunk(latent_chunk_kernel<8, false>);
  else chunk(latent_chunk_kernel<16, false>);
  int parts = (int)(2 * 148 / ((long long)row_groups * a.heads > 2 * 148 ? 2 * 148 : (long long)row_groups * a.heads));
  const int most = (a.vdim + 7) / 8;
  parts = parts < 1 ? 1 : parts > most ? most : parts > 8 ? 8 : parts;
  const size_t j_smem = (size_t)LD_ROWS * (((g.rank + 7) & ~7) + g.splits) * sizeof(float);
  auto join = [&](auto kernel) {
    if (j_smem > 48 * 1024)
      LB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)j_smem));
    launch_pdl(kernel, dim3((unsigned)a.heads, (unsigned)parts, row_groups), dim3(LD_THREADS), j_smem, st, g_pdl_enabled, g,
               (const float *)po, (const float2 *)ml, static_cast<const bf16 *>(a.w_uv), a.w_ld, rows,
               static_cast<bf16 *>(a.out), a.out_ld);
  };
  if (g.rank <= 256) join(latent_join_kernel<1>);
  else if (g.rank <= 512) join(latent_join_kernel<2>);
  else join(latent_join_kernel<4>);
  return 3;
}

}  // namespace lb
