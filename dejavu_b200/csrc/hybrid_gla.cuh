// Arguments and device helpers shared by the gated linear attention kernels.
#pragma once
#include "mma.cuh"

namespace djv {

constexpr int GLA_THREADS = 256;

struct GlaArgs {
  void *out;
  const void *proj;
  long long ld;
  const float *a2, *a2_bias, *norm;
  float inv_tau, eps, scale;
  float *state;
  const long long *pos;
  int B, n, H, dk, dv, rank;
  int C, nc;      // chunk length, number of chunks
  float *contrib; // (B, H, nc, dk, dv): contributions, then incoming states
  float *decay;   // (B, H, nc, dk): B_C
  float *cum;     // (B*n, H, dk): B_t
};

// tensor-core form of the chunk kernels (bf16); chunks of GLA_MMA_CHUNK tokens
constexpr int GLA_MMA_CHUNK = 64;
bool gla_mma_supported(int dtype, int dk, int dv);
int gla_mma_chunk_state(const GlaArgs &a, cudaStream_t st);
int gla_mma_chunk_out(const GlaArgs &a, cudaStream_t st);

}  // namespace djv
