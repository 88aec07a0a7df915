// Arguments shared by the kernels of the routed feed-forward.
#pragma once
#include "rowdot.cuh"

namespace djv {

// One grouped matrix product over rows sorted by expert: rows offsets[e] .. offsets[e+1] - 1 of x times w[e].
struct GroupedArgs {
  void *y;             // (R, N) of T, or (R, N / 2) behind the gated unit
  const void *x;       // (R, K)
  const void *w;       // (E, N, K); behind the gated unit rows 2i, 2i + 1 of an expert are gate and up of output i
  const float *scale;  // (R): factor on the product's rows, before the unit; null: 1
  const int *offsets;  // (E + 1)
  int R, E, N, K;
  int glu;
};

// (expert, first row) of row tile `tile` when every expert's rows are cut into tiles of `rows`; false past the last one
__device__ __forceinline__ bool grouped_tile(const int *offsets, int E, int rows, int tile, int &e, int &r0, int &r1) {
  int left = tile;
  for (e = 0; e < E; ++e) {
    r0 = offsets[e];
    r1 = offsets[e + 1];
    const int t = (r1 - r0 + rows - 1) / rows;
    if (left < t) {
      r0 += left * rows;
      return true;
    }
    left -= t;
  }
  return false;
}

// tensor-core form (bf16)
bool moe_grouped_tc_supported(int dtype, const GroupedArgs &a);
int moe_grouped_tc(const GroupedArgs &a, cudaStream_t st);

}  // namespace djv
