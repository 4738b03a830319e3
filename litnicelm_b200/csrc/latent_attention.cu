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
//                                side by side for the expanding kernels (latent_attention_tc.cu)
//   latent_attention_rows_kernel any size, one CTA per row and head, float or bfloat16 storage
//   latent_query / latent_chunk / latent_join   few rows on bfloat16: the absorbed query per head; key
//                                chunks of 64 for 16 heads at a time on mma.sync tiles, the fp32 query
//                                and weights entering as two bfloat16 terms each; the join of the chunks
//                                followed by W_uv
// Scores, weights and norms are 32-bit throughout.
#include "model.cuh"

#include <cuda_bf16.h>

namespace lb {

namespace {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void put(float *p, float v) { *p = v; }
__device__ __forceinline__ void put(bf16 *p, float v) { *p = __float2bfloat16_rn(v); }

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

// One warp per position: positions first .. p0 + n - 1 (first <= p0) of stream b. Old positions are
// copied from the cache to the packed rows, new ones normalised (dkv given) or, for a layer that uses
// another layer's latents, copied as well.
template <typename T>
__global__ void __launch_bounds__(128)
latent_store_kernel(const float *__restrict__ dkv, int dkv_ld, const float *__restrict__ gain, float eps, T *__restrict__ cache,
                    int cap, int ld, int rank, T *__restrict__ packed, int packed_rows, int first, int n, int p0_host,
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
  const float *src = dkv + ((long long)b * n + (p - p0)) * dkv_ld;
  float s = 0.f;
  for (int c = lane; c < rank; c += 32) s = fmaf(src[c], src[c], s);
  const float inv = 1.0f / sqrtf(warp_sum(s) / (float)rank + eps);
  for (int c = lane; c < ld; c += 32) {
    const float v = c < rank ? src[c] * inv * gain[c] : 0.f;
    put(row + c, v);
    if (dst) put(dst + c, v);
  }
}

// ---- any size ------------------------------------------------------------------

constexpr int LR_THREADS = 256;
constexpr int LR_KEYS = 64;  // keys per pass

template <typename T>
__global__ void __launch_bounds__(LR_THREADS)
latent_attention_rows_kernel(const T *__restrict__ q, int q_ld, const T *__restrict__ w_uk, const T *__restrict__ w_uv,
                             int w_ld, const T *__restrict__ cache, int cap, int ld, int rank, int dim, int vdim, float scale,
                             int window, T *__restrict__ out, int out_ld, int n, int p0_host, const LoopState *state,
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

constexpr int LD_KEYS = 64;      // keys per chunk
constexpr int LD_HEADS = 16;     // heads per CTA: the rows of an mma tile
constexpr int LD_THREADS = 256;
constexpr int LQ_COLS = 64;      // latent columns per CTA of the query kernel
constexpr int LQ_ROWS = 4;       // rows per CTA of the query kernel
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
__device__ __forceinline__ void split2(float v, bf16 &hi, bf16 &lo) {
  hi = __float2bfloat16_rn(v);
  lo = __float2bfloat16_rn(v - __bfloat162float(hi));
}

// qa[r, h, c] = scale * log2(e) * sum_e q[r, h, e] W_uk[h, e, c]: LQ_COLS columns of one head for up to
// LQ_ROWS rows; the four thread groups of a CTA take quarters of e.
__global__ void __launch_bounds__(LD_THREADS)
latent_query_kernel(const bf16 *__restrict__ q, int q_ld, const bf16 *__restrict__ w_uk, int w_ld, int rank, int dim,
                    float factor, int heads, long long n_rows, float *__restrict__ qa) {
  __shared__ float part[4][LQ_ROWS][LQ_COLS];
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.y;
  const int cl = threadIdx.x & (LQ_COLS - 1), grp = threadIdx.x / LQ_COLS;
  const int c = blockIdx.x * LQ_COLS + cl;
  const long long r0 = (long long)blockIdx.z * LQ_ROWS;
  const int nr = (int)min((long long)LQ_ROWS, n_rows - r0);
  float acc[LQ_ROWS] = {};
  if (c < rank) {
    const int e0 = dim * grp / 4, e1 = dim * (grp + 1) / 4;
#pragma unroll 8
    for (int e = e0; e < e1; ++e) {
      const float w = to_f(w_uk[((long long)h * dim + e) * w_ld + c]);
#pragma unroll
      for (int i = 0; i < LQ_ROWS; ++i)
        if (i < nr) acc[i] = fmaf(to_f(q[(r0 + i) * q_ld + (long long)h * dim + e]), w, acc[i]);
    }
  }
#pragma unroll
  for (int i = 0; i < LQ_ROWS; ++i) part[grp][i][cl] = acc[i];
  __syncthreads();
  // thread group i sums row i
  if (grp < nr && c < rank)
    qa[((r0 + grp) * heads + h) * rank + c] =
        (part[0][grp][cl] + part[1][grp][cl] + part[2][grp][cl] + part[3][grp][cl]) * factor;
}

// Chunk blockIdx.x (LD_KEYS keys from the window's first one on) of row blockIdx.z for heads
// blockIdx.y * 16 ..: partial o[head][rank] = sum_j 2^(s_j - m) c_j with m, l = sum of the weights.
__global__ void __launch_bounds__(LD_THREADS)
latent_chunk_kernel(const float *__restrict__ qa, const bf16 *__restrict__ cache, int cap, int ld, int rank, int heads,
                    int window, int n, int p0_host, const LoopState *state, int slot0, float *__restrict__ part_o,
                    float2 *__restrict__ part_ml) {
  extern __shared__ __align__(16) unsigned char smraw[];
  const int rk = (rank + 15) & ~15, pitch = rk + 8;  // halves per row: 16-byte rows whose fragments hit distinct banks
  bf16 *ck = reinterpret_cast<bf16 *>(smraw);        // [LD_KEYS][pitch]
  bf16 *qh = ck + LD_KEYS * pitch;                   // [16][pitch] high and low terms of the query
  bf16 *ql = qh + LD_HEADS * pitch;
  constexpr int PP = LD_KEYS + 8;
  bf16 *ph = ql + LD_HEADS * pitch;                  // [16][PP] high and low terms of the weights
  bf16 *pl = ph + LD_HEADS * PP;
  float *sc = reinterpret_cast<float *>(pl + LD_HEADS * PP);  // [16][LD_KEYS + 4]
  constexpr int SP = LD_KEYS + 4;
  pdl_launch_dependents();
  pdl_wait();
  const long long r = blockIdx.z;
  const int b = (int)(r / n), t = (int)(r - (long long)b * n);
  const int p = (state ? state->s - n : p0_host) + t;
  const int lo = max(0, p - window + 1);
  const int j0 = lo + blockIdx.x * LD_KEYS;
  if (j0 > p) return;
  const int nk = min(LD_KEYS, p - j0 + 1);
  const int h0 = blockIdx.y * LD_HEADS, nh = min(LD_HEADS, heads - h0);
  const int tid = threadIdx.x, lane = tid & 31, wid = tid >> 5;
  const int g = lane >> 2, tq = lane & 3;
  const bf16 *src = cache + ((long long)(slot0 + b) * cap + j0) * ld;
  // latents: 16-byte pieces; the cache's rows end on a multiple of 8 columns with zeros behind the rank
  for (int i = tid; i < LD_KEYS * (rk / 8); i += LD_THREADS) {
    const int j = i / (rk / 8), c = (i - j * (rk / 8)) * 8;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (j < nk && c < ld) v = *reinterpret_cast<const uint4 *>(src + (long long)j * ld + c);
    *reinterpret_cast<uint4 *>(ck + j * pitch + c) = v;
  }
  for (int i = tid; i < LD_HEADS * rk; i += LD_THREADS) {
    const int hh = i / rk, c = i - hh * rk;
    const float v = hh < nh && c < rank ? qa[(r * heads + h0 + hh) * rank + c] : 0.f;
    bf16 hi, low;
    split2(v, hi, low);
    qh[hh * pitch + c] = hi;
    ql[hh * pitch + c] = low;
  }
  __syncthreads();
  {  // scores: warp w takes keys 8w .. 8w + 7
    float d[4] = {0.f, 0.f, 0.f, 0.f};
    const bf16 *kr = ck + (wid * 8 + g) * pitch + tq * 2;
    const bf16 *ah = qh + g * pitch + tq * 2, *al = ql + g * pitch + tq * 2;
    for (int k = 0; k < rk; k += 16) {
      const unsigned b0 = *reinterpret_cast<const unsigned *>(kr + k), b1 = *reinterpret_cast<const unsigned *>(kr + k + 8);
      const unsigned a[4] = {*reinterpret_cast<const unsigned *>(ah + k), *reinterpret_cast<const unsigned *>(ah + k + 8 * pitch),
                             *reinterpret_cast<const unsigned *>(ah + k + 8),
                             *reinterpret_cast<const unsigned *>(ah + k + 8 * pitch + 8)};
      const unsigned a2[4] = {*reinterpret_cast<const unsigned *>(al + k), *reinterpret_cast<const unsigned *>(al + k + 8 * pitch),
                              *reinterpret_cast<const unsigned *>(al + k + 8),
                              *reinterpret_cast<const unsigned *>(al + k + 8 * pitch + 8)};
      mma_bf16(d, a2, b0, b1);
      mma_bf16(d, a, b0, b1);
    }
    const int j = wid * 8 + tq * 2;
    sc[g * SP + j] = d[0];
    sc[g * SP + j + 1] = d[1];
    sc[(g + 8) * SP + j] = d[2];
    sc[(g + 8) * SP + j + 1] = d[3];
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 2; ++i) {  // weights: warp w takes heads 2w and 2w + 1, a lane two keys
    const int hh = wid * 2 + i;
    const float s0 = lane < nk ? sc[hh * SP + lane] : -INFINITY;
    const float s1 = lane + 32 < nk ? sc[hh * SP + lane + 32] : -INFINITY;
    const float m = warp_max(fmaxf(s0, s1));
    const float p0 = exp2f(s0 - m), p1 = exp2f(s1 - m);
    const float l = warp_sum(p0 + p1);
    bf16 hi, low;
    split2(p0, hi, low);
    ph[hh * PP + lane] = hi;
    pl[hh * PP + lane] = low;
    split2(p1, hi, low);
    ph[hh * PP + lane + 32] = hi;
    pl[hh * PP + lane + 32] = low;
    if (lane == 0 && hh < nh) part_ml[(r * heads + h0 + hh) * gridDim.x + blockIdx.x] = make_float2(m, l);
  }
  __syncthreads();
  unsigned a[LD_KEYS / 16][4], a2[LD_KEYS / 16][4];
#pragma unroll
  for (int k = 0; k < LD_KEYS / 16; ++k) {
    const bf16 *x = ph + g * PP + tq * 2 + k * 16, *y = pl + g * PP + tq * 2 + k * 16;
    a[k][0] = *reinterpret_cast<const unsigned *>(x);
    a[k][1] = *reinterpret_cast<const unsigned *>(x + 8 * PP);
    a[k][2] = *reinterpret_cast<const unsigned *>(x + 8);
    a[k][3] = *reinterpret_cast<const unsigned *>(x + 8 * PP + 8);
    a2[k][0] = *reinterpret_cast<const unsigned *>(y);
    a2[k][1] = *reinterpret_cast<const unsigned *>(y + 8 * PP);
    a2[k][2] = *reinterpret_cast<const unsigned *>(y + 8);
    a2[k][3] = *reinterpret_cast<const unsigned *>(y + 8 * PP + 8);
  }
  for (int c0 = wid * 8; c0 < rk; c0 += LD_THREADS / 32 * 8) {
    float d[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int k = 0; k < LD_KEYS / 16; ++k) {
      unsigned b0, b1;
      ldmatrix_x2_trans(b0, b1, ck + (k * 16 + (lane & 15)) * pitch + c0);
      mma_bf16(d, a2[k], b0, b1);
      mma_bf16(d, a[k], b0, b1);
    }
    const int c = c0 + tq * 2;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int hh = g + 8 * i;
      if (hh >= nh) continue;
      float *o = part_o + ((r * heads + h0 + hh) * gridDim.x + blockIdx.x) * (long long)rank;
      if (c < rank) o[c] = d[2 * i];
      if (c + 1 < rank) o[c + 1] = d[2 * i + 1];
    }
  }
}

// Joins the chunks of one row and head and maps the weighted latent through W_uv; the CTAs of grid.y
// share the head's value rows.
__global__ void __launch_bounds__(LD_THREADS)
latent_join_kernel(const float *__restrict__ part_o, const float2 *__restrict__ part_ml, int chunks, const bf16 *__restrict__ w_uv,
                   int w_ld, int rank, int vdim, int heads, int window, int n, int p0_host, const LoopState *state,
                   bf16 *__restrict__ out, int out_ld) {
  extern __shared__ float ol[];  // [rank rounded up to 8] weighted latent, then [chunks] factors
  pdl_launch_dependents();
  pdl_wait();
  const int h = blockIdx.x, lane = threadIdx.x & 31, wid = threadIdx.x >> 5;
  const long long r = blockIdx.z;
  const int t = (int)(r % n);
  const int p = (state ? state->s - n : p0_host) + t;
  const int nc = (min(window, p + 1) + LD_KEYS - 1) / LD_KEYS;
  const int r8 = (rank + 7) & ~7;
  float *fac = ol + r8;
  const float2 *ml = part_ml + (r * heads + h) * chunks;
  float m = -INFINITY, l = 0.f;
  for (int c = lane; c < nc; c += 32) m = fmaxf(m, ml[c].x);
  m = warp_max(m);
  for (int c = lane; c < nc; c += 32) l += ml[c].y * exp2f(ml[c].x - m);
  l = warp_sum(l);
  if (wid == 0)
    for (int c = lane; c < nc; c += 32) fac[c] = exp2f(ml[c].x - m) / l;
  __syncthreads();
  const float *o = part_o + (r * heads + h) * (long long)chunks * rank;
  for (int c = threadIdx.x; c < r8; c += LD_THREADS) {
    float a = 0.f;
    if (c < rank) {
#pragma unroll 4
      for (int i = 0; i < nc; ++i) a = fmaf(fac[i], o[(long long)i * rank + c], a);
    }
    ol[c] = a;
  }
  __syncthreads();
  const int e_per = (vdim + gridDim.y - 1) / gridDim.y;
  const int e1 = min(vdim, (int)(blockIdx.y + 1) * e_per);
  for (int e = blockIdx.y * e_per + wid; e < e1; e += LD_THREADS / 32) {
    const bf16 *wr = w_uv + ((long long)h * vdim + e) * w_ld;
    float s = 0.f;
    for (int c = lane * 8; c < r8; c += 256) {  // rows of W_uv end on a multiple of 8 with zeros behind the rank
      const uint4 v = *reinterpret_cast<const uint4 *>(wr + c);
      const unsigned u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        s = fmaf(__uint_as_float(u[i] << 16), ol[c + 2 * i], s);
        s = fmaf(__uint_as_float(u[i] & 0xffff0000u), ol[c + 2 * i + 1], s);
      }
    }
    s = warp_sum(s);
    if (lane == 0) out[r * out_ld + (long long)h * vdim + e] = __float2bfloat16_rn(s);
  }
}

size_t chunk_smem(int rank) {
  const int pitch = ((rank + 15) & ~15) + 8;
  return (size_t)(LD_KEYS + 2 * LD_HEADS) * pitch * 2 + (size_t)2 * LD_HEADS * (LD_KEYS + 8) * 2 +
         (size_t)LD_HEADS * (LD_KEYS + 4) * 4;
}
int chunks_of(int window, int s_cap) { return ((window < s_cap ? window : s_cap) + LD_KEYS - 1) / LD_KEYS; }

}  // namespace

void launch_latent_store(const float *dkv, int dkv_ld, const float *gain, float eps, const LatentCache &cache,
                         void *packed, int packed_rows, int first, Precision type, const RowBatch &b, cudaStream_t st) {
  const int count = packed ? b.p0 + b.n - first : b.n;
  const dim3 grid((unsigned)((count + 3) / 4), (unsigned)b.streams);
  if (type == Precision::BF16)
    launch_pdl(latent_store_kernel<bf16>, grid, dim3(128), 0, st, g_pdl_enabled, dkv, dkv_ld, gain, eps,
               static_cast<bf16 *>(cache.rows), cache.cap, cache.ld, cache.rank, static_cast<bf16 *>(packed), packed_rows,
               first, b.n, b.p0, b.state, b.slot0);
  else
    launch_pdl(latent_store_kernel<float>, grid, dim3(128), 0, st, g_pdl_enabled, dkv, dkv_ld, gain, eps,
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

bool latent_decode_supports(const LatentAttention &a) { return chunk_smem(a.cache.rank) <= 220 * 1024; }

size_t latent_decode_scratch_floats(int heads, int rank, int window, int s_cap, long long rows) {
  const size_t rh = (size_t)rows * heads, c = (size_t)chunks_of(window, s_cap);
  return (rh * rank + 3) / 4 * 4 + rh * c * 2 + rh * c * rank;
}

int launch_latent_decode(const LatentAttention &a, float *scratch, const RowBatch &b, cudaStream_t st) {
  const long long rows = b.rows();
  const int rank = a.cache.rank, chunks = chunks_of(a.window, b.s_cap);
  float *qa = scratch;
  float2 *ml = reinterpret_cast<float2 *>(scratch + ((size_t)rows * a.heads * rank + 3) / 4 * 4);
  float *po = reinterpret_cast<float *>(ml + (size_t)rows * a.heads * chunks);
  launch_pdl(latent_query_kernel,
             dim3((unsigned)((rank + LQ_COLS - 1) / LQ_COLS), (unsigned)a.heads, (unsigned)((rows + LQ_ROWS - 1) / LQ_ROWS)),
             dim3(LD_THREADS), 0, st, g_pdl_enabled, static_cast<const bf16 *>(a.q), a.q_ld, static_cast<const bf16 *>(a.w_uk),
             a.w_ld, rank, a.dim, a.scale * LOG2E, a.heads, rows, qa);
  const size_t smem = chunk_smem(rank);
  if (smem > 48 * 1024)
    LB_CUDA(cudaFuncSetAttribute(latent_chunk_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  launch_pdl(latent_chunk_kernel,
             dim3((unsigned)chunks, (unsigned)((a.heads + LD_HEADS - 1) / LD_HEADS), (unsigned)rows), dim3(LD_THREADS), smem,
             st, g_pdl_enabled, (const float *)qa, static_cast<const bf16 *>(a.cache.rows), a.cache.cap, a.cache.ld, rank,
             a.heads, a.window, b.n, b.p0, b.state, b.slot0, po, ml);
  int parts = (int)(148 / (rows * a.heads > 148 ? 148 : rows * a.heads));
  const int most = (a.vdim + 7) / 8;
  parts = parts < 1 ? 1 : parts > most ? most : parts > 8 ? 8 : parts;
  launch_pdl(latent_join_kernel, dim3((unsigned)a.heads, (unsigned)parts, (unsigned)rows), dim3(LD_THREADS),
             ((size_t)((rank + 7) & ~7) + chunks) * sizeof(float), st, g_pdl_enabled, (const float *)po, (const float2 *)ml,
             chunks, static_cast<const bf16 *>(a.w_uv), a.w_ld, rank, a.vdim, a.heads, a.window, b.n, b.p0, b.state,
             static_cast<bf16 *>(a.out), a.out_ld);
  return 3;
}

}  // namespace lb
