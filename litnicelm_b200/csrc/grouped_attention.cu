// Softmax attention with shared key and value heads: query head h of the row at position p attends to the
// keys of group h / (heads / groups) at positions span.first(p) .. p.
//
//   qk_norm_rotate_kernel   RMS norm over a whole row of queries (and of keys), rotary positions, keys and
//                           values into the caches
//   grouped_rows_kernel     any number of rows, keys and values read once for up to eight query heads of a
//                           group; few rows: the keys are split over the CTAs of a cluster, whose partial
//                           results meet in shared memory
// (Many rows on tensor cores: prefill_attention_tc.cu.) Norms, angles, scores, weights and sums are 32-bit; the
// angle itself is reduced to one turn in double, so it does not lose digits far into a sequence.
#include "model.cuh"
#include "tc_ptx.cuh"

#include <cuda_bf16.h>

namespace lb {

namespace {

typedef __nv_bfloat16 bf16;

constexpr int GA_THREADS = 256;
constexpr int GA_KEYS = 128;    // keys per tile
constexpr int GA_CLUSTER = 8;   // CTAs of the largest cluster
constexpr float LOG2E = 1.4426950408889634f;

template <typename T>
struct Piece;  // 16 bytes of a row
template <>
struct Piece<bf16> {
  static constexpr int N = 8;
  uint4 u;
  __device__ __forceinline__ void load(const bf16 *p) { u = *reinterpret_cast<const uint4 *>(p); }
  __device__ __forceinline__ void unpack(float (&f)[8]) const {
    const unsigned w[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      f[2 * i] = __uint_as_float(w[i] << 16);
      f[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u);
    }
  }
  static __device__ __forceinline__ void store(bf16 *p, const float (&f)[8]) {
    unsigned w[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const __nv_bfloat162 v = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
      w[i] = *reinterpret_cast<const unsigned *>(&v);
    }
    *reinterpret_cast<uint4 *>(p) = make_uint4(w[0], w[1], w[2], w[3]);
  }
};
template <>
struct Piece<float> {
  static constexpr int N = 4;
  float4 u;
  __device__ __forceinline__ void load(const float *p) { u = *reinterpret_cast<const float4 *>(p); }
  __device__ __forceinline__ void unpack(float (&f)[4]) const {
    f[0] = u.x;
    f[1] = u.y;
    f[2] = u.z;
    f[3] = u.w;
  }
  static __device__ __forceinline__ void store(float *p, const float (&f)[4]) {
    *reinterpret_cast<float4 *>(p) = make_float4(f[0], f[1], f[2], f[3]);
  }
};

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

struct RowsShape {
  int n, p0, slot0;
  const LoopState *state;
  __device__ int position(long long r, int &b) const {
    b = (int)(r / n);
    return (state ? state->s - n : p0) + (int)(r - (long long)b * n);
  }
};

// One CTA per row. Shared memory: the row's queries and keys times their weights in 32-bit, then cosines and sines.
// FOUR: four neighbouring coordinates rotate (or pass) alike and stay within one half (rot.dims % 8 == 0).
template <typename T, bool FOUR>
__global__ void __launch_bounds__(GA_THREADS)
qk_norm_rotate_kernel(const T *src, int ld, const float *__restrict__ q_weight, const float *__restrict__ k_weight, float eps,
                      int q_cols, int k_cols, int v_cols, int dim, float q_count, float k_count, Rotation rot, T *q, int q_ld,
                      T *k_cache, T *v_cache, int cap, RowsShape g) {
  extern __shared__ __align__(16) float row[];
  __shared__ float part[2][GA_THREADS / 32];
  constexpr int P = Piece<T>::N;
  const int cols = q_cols + k_cols, half = rot.dims >> 1;
  float *cs = row + cols, *sn = cs + half;
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, wid = tid >> 5;
  const long long r = blockIdx.x;
  int b;
  const int p = g.position(r, b);
  const T *x = src + r * ld;
  const long long at = (long long)(g.slot0 + b) * cap + p;
  float sq = 0.f, sk = 0.f;
  for (int c = tid * P; c < cols; c += GA_THREADS * P) {
    Piece<T> v;
    v.load(x + c);
    const float *w = c < q_cols ? q_weight + c : k_weight + (c - q_cols);
    float f[P];
    v.unpack(f);
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < P; i += 4) {
      const float4 y = *reinterpret_cast<const float4 *>(w + i);
      s = fmaf(f[i], f[i], fmaf(f[i + 1], f[i + 1], fmaf(f[i + 2], f[i + 2], fmaf(f[i + 3], f[i + 3], s))));
      *reinterpret_cast<float4 *>(row + c + i) = make_float4(f[i] * y.x, f[i + 1] * y.y, f[i + 2] * y.z, f[i + 3] * y.w);
    }
    if (c < q_cols) sq += s;
    else sk += s;
  }
  for (int c = tid * P; c < v_cols; c += GA_THREADS * P) {
    Piece<T> v;
    v.load(x + cols + c);
    *reinterpret_cast<decltype(v.u) *>(v_cache + at * v_cols + c) = v.u;
  }
  for (int i = GA_THREADS - 1 - tid; i < half; i += GA_THREADS) {  // the last threads have the fewest pieces
    double t = (double)p * rot.turns[i];
    t -= 2.0 * rint(0.5 * t);
    float s, c;
    sincospif((float)t, &s, &c);
    cs[i] = c * rot.amplitude;
    sn[i] = s * rot.amplitude;
  }
  sq = warp_sum(sq);
  sk = warp_sum(sk);
  if (lane == 0) {
    part[0][wid] = sq;
    part[1][wid] = sk;
  }
  __syncthreads();
  sq = sk = 0.f;
#pragma unroll
  for (int i = 0; i < GA_THREADS / 32; ++i) {
    sq += part[0][i];
    sk += part[1][i];
  }
  const float iq = 1.0f / sqrtf(sq / q_count + eps), ik = 1.0f / sqrtf(sk / k_count + eps);
  auto four = [](const float *s) { return *reinterpret_cast<const float4 *>(s); };
  for (int c = tid * P; c < cols; c += GA_THREADS * P) {
    const bool is_q = c < q_cols;
    const float inv = is_q ? iq : ik;
    const int e0 = (is_q ? c : c - q_cols) % dim, h0 = c - e0;  // head's first column
    float f[P];
#pragma unroll
    for (int i = 0; i < P; i += FOUR ? 4 : 1) {
      const int e = e0 + i;
      if constexpr (FOUR) {
        float4 v = four(row + h0 + e);
        if (e < 2 * half) {
          const bool low = e < half;
          const float4 w = four(row + h0 + (low ? e + half : e - half)), y = four(cs + (low ? e : e - half));
          float4 z = four(sn + (low ? e : e - half));
          if (low) z = make_float4(-z.x, -z.y, -z.z, -z.w);
          v = make_float4(v.x * y.x + w.x * z.x, v.y * y.y + w.y * z.y, v.z * y.z + w.z * z.z, v.w * y.w + w.w * z.w);
        }
        f[i] = v.x * inv;
        f[i + 1] = v.y * inv;
        f[i + 2] = v.z * inv;
        f[i + 3] = v.w * inv;
      } else {
        float v = row[h0 + e];
        if (e < half) v = v * cs[e] - row[h0 + e + half] * sn[e];
        else if (e < 2 * half) v = v * cs[e - half] + row[h0 + e - half] * sn[e - half];
        f[i] = v * inv;
      }
    }
    Piece<T>::store(is_q ? q + r * q_ld + c : k_cache + at * k_cols + (c - q_cols), f);
  }
}

struct RowsArgs {
  int heads, groups, per, dim, vdim;
  float factor;  // scale * log2(e)
  KeySpan span;
  int q_ld, cap, out_ld;
  int splits, keys_per_split;
};

// Split blockIdx.x of the keys, R query heads of one group (blockIdx.y), row blockIdx.z.
template <typename T, int R>
__global__ void __launch_bounds__(GA_THREADS, R <= 4 ? 2 : 1)
grouped_rows_kernel(RowsArgs a, const T *q, const T *k_cache, const T *v_cache, T *out, RowsShape g) {
  constexpr int P = Piece<T>::N;
  extern __shared__ __align__(16) float sm[];
  float *qs = sm;                          // [R][dim] scaled queries
  float *sc = qs + R * a.dim;              // [R][GA_KEYS] scores, then weights
  float *red = sc + R * GA_KEYS;           // [key groups][vdim] partial sums of one head
  float *os = red + GA_THREADS * P;        // [R][vdim] this split's sums
  __shared__ float fac[R];
  __shared__ float2 ml[R];
  pdl_launch_dependents();
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, wid = tid >> 5;
  const long long r = blockIdx.z;
  const int blocks = (a.per + R - 1) / R;
  const int grp = blockIdx.y / blocks, hb = (blockIdx.y - grp * blocks) * R;
  const int h0 = grp * a.per + hb, nh = min(R, a.per - hb);
  int b;
  const int p = g.position(r, b);
  const int j0 = max(0, a.span.first(p)) + blockIdx.x * a.keys_per_split;
  const int total = max(0, min(a.keys_per_split, p - j0 + 1));
  const int k_ld = a.groups * a.dim, v_ld = a.groups * a.vdim;
  const T *kr = k_cache + ((long long)(g.slot0 + b) * a.cap + j0) * k_ld + grp * a.dim;
  const T *vr = v_cache + ((long long)(g.slot0 + b) * a.cap + j0) * v_ld + grp * a.vdim;
  // queries by planes of four elements of every piece: lanes on neighbouring pieces read neighbouring 16 bytes
  for (int i = tid; i < R * a.dim; i += GA_THREADS) {
    const int hh = i / a.dim, e = i - hh * a.dim;
    qs[hh * a.dim + (e % P / 4) * (a.dim / P * 4) + e / P * 4 + (e & 3)] =
        i < nh * a.dim ? to_f(q[r * a.q_ld + (long long)h0 * a.dim + i]) * a.factor : 0.f;
  }
  const int pieces = a.dim / P, cols = a.vdim / P;       // 16-byte pieces of a key and of a value
  const int key_groups = GA_THREADS / cols;
  const int vc = tid % cols * P, vg = tid / cols;        // this thread's value columns and its key group
  const bool summing = vg < key_groups;
  float acc[R][P];
#pragma unroll
  for (int h = 0; h < R; ++h)
#pragma unroll
    for (int i = 0; i < P; ++i) acc[h][i] = 0.f;
  float m = -INFINITY, l = 0.f;  // of head wid, in every lane of its warp
  __syncthreads();
  for (int k0 = 0; k0 < total; k0 += GA_KEYS) {
    const int nk = min(GA_KEYS, total - k0);
    {  // scores: eight lanes per key, batches of four keys per warp
      constexpr int BATCHES = GA_KEYS / (GA_THREADS / 8);
      const int sub = lane & 7, j0w = wid * (GA_KEYS / (GA_THREADS / 32)) + (lane >> 3);
      const T *kp[BATCHES];
      float sum[BATCHES][R];
#pragma unroll
      for (int i = 0; i < BATCHES; ++i) {
        kp[i] = kr + (long long)(k0 + min(j0w + 4 * i, nk - 1)) * k_ld;
#pragma unroll
        for (int h = 0; h < R; ++h) sum[i][h] = 0.f;
      }
      for (int c = sub; c < pieces; c += 8) {
        Piece<T> x[BATCHES];
#pragma unroll
        for (int i = 0; i < BATCHES; ++i) x[i].load(kp[i] + c * P);
        float f[BATCHES][P];
#pragma unroll
        for (int i = 0; i < BATCHES; ++i) x[i].unpack(f[i]);
#pragma unroll
        for (int h = 0; h < R; ++h) {
          const float *qh = qs + h * a.dim + c * 4;
#pragma unroll
          for (int e = 0; e < P; e += 4) {
            const float4 w = *reinterpret_cast<const float4 *>(qh + e * pieces);
#pragma unroll
            for (int i = 0; i < BATCHES; ++i)
              sum[i][h] = fmaf(f[i][e], w.x, fmaf(f[i][e + 1], w.y, fmaf(f[i][e + 2], w.z, fmaf(f[i][e + 3], w.w, sum[i][h]))));
          }
        }
      }
#pragma unroll
      for (int o = 4; o > 0; o >>= 1)
#pragma unroll
        for (int h = 0; h < R; ++h)
#pragma unroll
          for (int i = 0; i < BATCHES; ++i) sum[i][h] += __shfl_xor_sync(0xffffffffu, sum[i][h], o);
      if (sub == 0) {
#pragma unroll
        for (int h = 0; h < R; ++h)
#pragma unroll
          for (int i = 0; i < BATCHES; ++i) {
            const int j = j0w + 4 * i;
            sc[h * GA_KEYS + j] = j < nk ? sum[i][h] : -INFINITY;
          }
      }
    }
    constexpr int PRE = 4;  // values on their way under the softmax
    Piece<T> pre[PRE];
#pragma unroll
    for (int i = 0; i < PRE; ++i)
      pre[i].load(vr + (long long)(k0 + min(vg + i * key_groups, nk - 1)) * v_ld + (summing ? vc : 0));
    __syncthreads();
    if (wid < R) {  // weights: a lane takes four keys
      float4 *s = reinterpret_cast<float4 *>(sc + wid * GA_KEYS) + lane;
      float4 v = *s;
      const float mn = fmaxf(m, warp_max(fmaxf(fmaxf(v.x, v.y), fmaxf(v.z, v.w))));
      v = make_float4(exp2f(v.x - mn), exp2f(v.y - mn), exp2f(v.z - mn), exp2f(v.w - mn));
      const float keep = exp2f(m - mn);
      l = l * keep + warp_sum((v.x + v.y) + (v.z + v.w));
      m = mn;
      *s = v;
      if (lane == 0) fac[wid] = keep;
    }
    __syncthreads();
    if (summing) {
#pragma unroll
      for (int h = 0; h < R; ++h) {
        const float f = fac[h];
#pragma unroll
        for (int i = 0; i < P; ++i) acc[h][i] *= f;
      }
      auto add = [&](int j, const Piece<T> &v) {
        float f[P];
        v.unpack(f);
#pragma unroll
        for (int h = 0; h < R; ++h) {
          const float w = sc[h * GA_KEYS + j];
#pragma unroll
          for (int i = 0; i < P; ++i) acc[h][i] = fmaf(w, f[i], acc[h][i]);
        }
      };
#pragma unroll
      for (int i = 0; i < PRE; ++i)
        if (vg + i * key_groups < nk) add(vg + i * key_groups, pre[i]);
      for (int j = vg + PRE * key_groups; j < nk; j += key_groups) {
        Piece<T> v;
        v.load(vr + (long long)(k0 + j) * v_ld + vc);
        add(j, v);
      }
    }
    __syncthreads();
  }
  if (wid < R && lane == 0) ml[wid] = make_float2(m, l);
#pragma unroll
  for (int h = 0; h < R; ++h) {  // the key groups' sums, one head at a time
    if (summing) {
#pragma unroll
      for (int i = 0; i < P; ++i) red[vg * a.vdim + vc + i] = acc[h][i];
    }
    __syncthreads();
    for (int e = tid; e < a.vdim; e += GA_THREADS) {
      float s = 0.f;
      for (int k = 0; k < key_groups; ++k) s += red[k * a.vdim + e];
      os[h * a.vdim + e] = s;
    }
    __syncthreads();
  }
  T *o = out + r * a.out_ld + (long long)h0 * a.vdim;
  if (a.splits == 1) {
    for (int e = tid; e < nh * a.vdim; e += GA_THREADS) put(o + e, os[e] / ml[e / a.vdim].y);
    return;
  }
  __syncwarp();
  cluster_sync_all();
  const unsigned os_at = smem_u32(os), ml_at = smem_u32(ml);
  for (int e = blockIdx.x * GA_THREADS + tid; e < nh * a.vdim; e += a.splits * GA_THREADS) {
    const unsigned mine = ml_at + (unsigned)(e / a.vdim) * 8u;
    float mq[GA_CLUSTER], top = -INFINITY, sum = 0.f, v = 0.f;
#pragma unroll
    for (int i = 0; i < GA_CLUSTER; ++i) {
      mq[i] = i < a.splits ? ld_cluster_f32(cluster_map(mine, (unsigned)i)) : -INFINITY;
      top = fmaxf(top, mq[i]);
    }
#pragma unroll
    for (int i = 0; i < GA_CLUSTER; ++i) {
      if (i < a.splits) {
        const float f = exp2f(mq[i] - top);
        sum = fmaf(f, ld_cluster_f32(cluster_map(mine + 4u, (unsigned)i)), sum);
        v = fmaf(f, ld_cluster_f32(cluster_map(os_at + (unsigned)e * 4u, (unsigned)i)), v);
      }
    }
    put(o + e, v / sum);
  }
  __syncwarp();
  cluster_sync_all();  // a split's shared memory stays until every other has read it
}

template <typename T, int R>
void rows_launch(const RowsArgs &a, const GroupedAttention &at, const RowBatch &b, cudaStream_t st) {
  constexpr int P = Piece<T>::N;
  const size_t smem = ((size_t)R * (a.dim + GA_KEYS + a.vdim) + (size_t)GA_THREADS * P) * sizeof(float);
  auto kernel = grouped_rows_kernel<T, R>;
  if (smem > 40 * 1024) LB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  const dim3 grid((unsigned)a.splits, (unsigned)(a.groups * ((a.per + R - 1) / R)), (unsigned)b.rows());
  launch_pdl_cluster_x(kernel, grid, dim3(GA_THREADS), smem, st, g_pdl_enabled, (unsigned)a.splits, a,
                       static_cast<const T *>(at.q), static_cast<const T *>(at.k_cache), static_cast<const T *>(at.v_cache),
                       static_cast<T *>(at.out), RowsShape{b.n, b.p0, b.slot0, b.state});
}

template <typename T>
void rows_launch_t(const RowsArgs &a, const GroupedAttention &at, const RowBatch &b, cudaStream_t st) {
  if (a.per <= 1) rows_launch<T, 1>(a, at, b, st);
  else if (a.per <= 2) rows_launch<T, 2>(a, at, b, st);
  else if (a.per <= 4) rows_launch<T, 4>(a, at, b, st);
  else rows_launch<T, 8>(a, at, b, st);
}

template <typename T>
void norm_rotate_t(const void *src, int ld, const float *qw, const float *kw, float eps, int true_dim, const Rotation &rot,
                   const GroupedAttention &a, void *q, const RowBatch &b, cudaStream_t st) {
  const int qc = a.heads * a.dim, kc = a.groups * a.dim;
  const size_t smem = (size_t)(qc + kc + rot.dims) * sizeof(float);
  auto kernel = rot.dims % 8 == 0 ? qk_norm_rotate_kernel<T, true> : qk_norm_rotate_kernel<T, false>;
  if (smem > 40 * 1024) LB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  launch_pdl(kernel, dim3((unsigned)b.rows()), dim3(GA_THREADS), smem, st, g_pdl_enabled, static_cast<const T *>(src), ld, qw,
             kw, eps, qc, kc, a.groups * a.vdim, a.dim, (float)(a.heads * true_dim), (float)(a.groups * true_dim), rot,
             static_cast<T *>(q), a.q_ld, static_cast<T *>(a.k_cache), static_cast<T *>(a.v_cache), a.cap,
             RowsShape{b.n, b.p0, b.slot0, b.state});
}

}  // namespace

void launch_qk_norm_rotate(const void *src, int ld, const float *q_weight, const float *k_weight, float eps, int true_dim,
                           const Rotation &rot, const GroupedAttention &a, void *q, Precision type, const RowBatch &b,
                           cudaStream_t st) {
  if (type == Precision::BF16) norm_rotate_t<bf16>(src, ld, q_weight, k_weight, eps, true_dim, rot, a, q, b, st);
  else norm_rotate_t<float>(src, ld, q_weight, k_weight, eps, true_dim, rot, a, q, b, st);
}

void launch_grouped_attention_rows(const GroupedAttention &at, Precision type, const RowBatch &b, cudaStream_t st) {
  RowsArgs a{};
  a.heads = at.heads;
  a.groups = at.groups;
  a.per = at.heads / at.groups;
  a.dim = at.dim;
  a.vdim = at.vdim;
  a.factor = at.scale * LOG2E;
  a.span = at.span;
  a.q_ld = at.q_ld;
  a.cap = at.cap;
  a.out_ld = at.out_ld;
  // as many splits as keep every CTA resident (two per SM), no split without a tile of its own
  const int keys = at.span.size < b.s_cap ? at.span.size : b.s_cap, tiles = (keys + GA_KEYS - 1) / GA_KEYS;
  const long long ctas = b.rows() * at.groups * ((a.per + 7) / 8), room = 2 * 148 / ctas;
  int want = room < 1 ? 1 : room > GA_CLUSTER ? GA_CLUSTER : (int)room;
  if (want > tiles) want = tiles;
  const int tiles_per = (tiles + want - 1) / want;
  a.keys_per_split = tiles_per * GA_KEYS;
  a.splits = (tiles + tiles_per - 1) / tiles_per;
  if (type == Precision::BF16) rows_launch_t<bf16>(a, at, b, st);
  else rows_launch_t<float>(a, at, b, st);
}

}  // namespace lb
