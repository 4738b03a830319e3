// Device and host pieces that the two forms of the gated delta rule share (delta.cu, delta_chunk.cu).
#pragma once

#include <cuda_bf16.h>

#include "activation.cuh"
#include "model.cuh"

namespace lb {

constexpr float DELTA_UNIT_EPS = 1e-6f;

struct DeltaRows {
  int n, p0, slot0;
  const LoopState *state;
  __device__ __forceinline__ int first_position() const { return state ? state->s - n : p0; }
};

// Logarithm of a head's decay at a token (bounded, so that sums of a chunk stay finite; e^-10000 is zero in 32-bit).
__device__ __forceinline__ float delta_log_decay(float a, float a_log, float dt_bias) {
  return fmaxf(-expf(a_log) * softplus_f32(a + dt_bias), -1.0e4f);
}

constexpr int DELTA_CHUNK = 64;  // tokens per chunk of the chunked form

// What the scan of a portion's chunks reads: the convolved rows [rows][channels], and per stream, head and chunk the
// matrices [inverse high, low, A high, low][64][64] and the tokens' factors [e^G r, e^G r', e^(G_last - G) r, e^G_last][64].
struct DeltaChunks {
  int heads, groups, dim, vdim, channels, n, chunks;
  const __nv_bfloat16 *conv;
  __nv_bfloat16 *mats;
  float *factors;
};

// delta_chunk.cu: the recurrence of many rows on bfloat16 in chunks of 64 tokens. conv: the convolved rows
// [rows][conv_channels]. The output's norm and gate are applied where one CTA holds a whole head; otherwise
// o [rows][heads * vdim] is left in float.
bool delta_chunk_supports(const DeltaMixer &m);
size_t delta_chunk_bytes(const DeltaMixer &m, long long rows, int streams);
// Returns the kernels launched; *normed: whether m.out is written.
int launch_delta_chunks(const DeltaMixer &m, const void *conv, float *o, void *scratch, const RowBatch &b, bool *normed,
                        cudaStream_t st, DevErr *err);
// delta_scan_tc.cu: the scan on the sm_100a tensor cores; returns whether the norm and gate are applied.
bool delta_scan_tc_supports(const DeltaMixer &m);
bool launch_delta_scan_tc(const DeltaMixer &m, const DeltaChunks &c, float *o, const RowBatch &b, cudaStream_t st, DevErr *err);

}  // namespace lb
