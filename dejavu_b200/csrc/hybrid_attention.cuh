// Arguments shared by the sliding-window attention kernels.
#pragma once
#include "common.cuh"

namespace djv {

struct WindowArgs {
  void *out;              // (B*n, H*dv)
  const void *qkv;        // rows of q (H, dk) | k (G, dk) | v (G, dv)
  long long ld;
  const void *k_ring, *v_ring;
  const float *sink;      // (H) or null
  const long long *pos;   // (B) position of each sequence's first token of the call
  int B, n, H, G, dk, dv, cap, window;
  float scale;
};

// tensor-core form for prompt portions (bf16)
bool window_prefill_supported(const WindowArgs &a);
int window_prefill(const WindowArgs &a, cudaStream_t st);

}  // namespace djv
