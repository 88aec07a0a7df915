// Arguments shared by the windowed attention kernels.
#pragma once
#include "common.cuh"

namespace djv {

struct WindowArgs {
  void *out;              // (B*n, H*dv)
  const void *q;          // (B*n) rows of (H, dk)
  long long ldq;
  const void *k;          // rows of (G, dk - rot): the portion's own keys, and `past` rows of earlier tokens before them
  long long ldk;
  const void *v;          // rows of (G, dv), as the keys
  long long ldv;
  const void *tail;       // rows of `rot`: the last dimensions of a key where all heads share them, as the keys
  long long ldt;
  int rot;
  const void *gate;       // (B*n) rows of (H, dv), or null: outputs times sigmoid(gate)
  long long ldg;
  const void *k_ring, *v_ring;  // (B, G, cap, dk / dv): earlier tokens, or null: only the `past` rows
  const float *sink;      // (H) or null
  const long long *pos;   // (B) position of each sequence's first token of the call
  int B, n, H, G, dk, dv, cap, past, window;
  float scale;
};

// rows of k, v and tail: sequence b's token t (t < 0: before the portion) is row b * (past + n) + past + t
int window_attn_portion(int dtype, const WindowArgs &a, cudaStream_t st);

// tensor-core form for prompt portions (bf16)
bool window_prefill_supported(const WindowArgs &a);
int window_prefill(const WindowArgs &a, cudaStream_t st);

}  // namespace djv
