// Arguments shared by the decode kernels of latent attention.
#pragma once
#include "dtype.cuh"

namespace djv {

struct LatentDecodeArgs {
  void *out;           // (B, H * dv)
  void *qc;            // (B, H, rank + rot): queries against the ring's rows
  float *part_o;       // (B, H, splits, rank): sums of latents over a part of the window, weights e^(score - m)
  float *part_ml;      // (B, H, splits, 2): m, and the sum of the weights
  const void *proj;    // rows of q (H, dim + rot) | latent (rank) | shared key part (rot), neither normed nor rotated
  long long ld;
  const void *uk, *uv; // (H * dim, rank), (H * dv, rank)
  const float *norm;   // (rank)
  float eps;
  const float *freqs;  // (rot / 2)
  void *ring;          // (B, cap, rank + rot)
  const void *gate;    // rows of (H, dv), or null
  long long ldg;
  const long long *pos;
  int B, H, dim, rot, dv, rank, cap, window, splits;
  float scale;
};

constexpr int LQ_THREADS = 128, LQ_COLS = 64, LQ_REG = 8;
constexpr int LD_MAX_SPLITS = 32;

// parts the window is cut into
int latent_splits(int B, int H, int window);

// attention over the latents on the tensor cores (bf16)
bool latent_attend_mma_supported(const LatentDecodeArgs &a, bool bf16_rows);
int latent_attend_mma(const LatentDecodeArgs &a, cudaStream_t st);

}  // namespace djv
