// rowdot: y[b, m] = act(w[idx[m], :] . x[b, :] + bias[idx[m]]) for a few rows of x on the CUDA cores, for fp16, bf16
// and fp32 weights. Bound by HBM: every row of w is read exactly once.
#pragma once
#include "dtype.cuh"

namespace djv {

// Gated unit with a clamp: the gate is cut from above, the linear part on both sides, and one is added to it.
__device__ __forceinline__ float clamped_glu(float gate, float up, float limit) {
  const float g = fminf(gate, limit);
  const float u = fminf(fmaxf(up, -limit), limit);
  return g * sigmoid_f(1.702f * g) * (u + 1.f);
}

__device__ __forceinline__ float silu_glu(float gate, float up) { return gate * sigmoid_f(gate) * up; }

// gated units: two rows of the matrix make one output
__host__ __device__ constexpr bool is_glu(int act) { return act == DJV_ACT_CLAMPED_GLU || act == DJV_ACT_SILU_GLU; }
template <int ACT>
__device__ __forceinline__ float apply_glu(float gate, float up, float p) {
  return ACT == DJV_ACT_CLAMPED_GLU ? clamped_glu(gate, up, p) : silu_glu(gate, up);
}

// activations that take a constant, next to those that do not
template <int ACT>
__device__ __forceinline__ float apply_act_param(float v, float p) {
  if (ACT == DJV_ACT_SOFTCAP) return p * tanhf(v / p);
  return apply_act<ACT>(v);
}

// -------------------------------------------------------------------------------------------
// rowdot. A block has 8 warps split into 8/WPR groups of WPR warps; a group owns ROWS rows at a
// time and its 32*WPR lanes stride over the 16-byte chunks of those rows, U chunks in flight per
// lane per row. x is read through L1 (it is tiny and reused by every warp); weights bypass L1.
// Small M uses large WPR so that the whole device has loads in flight for a handful of rows.
// -------------------------------------------------------------------------------------------
constexpr int RD_THREADS = 256;
constexpr int RD_WARPS = RD_THREADS / WARP;

template <typename T, typename TO, int B, int ACT, int WPR, int ROWS, int U>
__global__ void __launch_bounds__(RD_THREADS)
rowdot_kernel(TO *__restrict__ Y, const T *__restrict__ W, const T *__restrict__ X,
              const void *__restrict__ idx, const T *__restrict__ bias, int M, int N,
              long long ldw, int idx64, int early, float act_param) {
  static_assert(!is_glu(ACT) || ROWS % 2 == 0, "a group owns whole (gate, up) pairs of rows");
  constexpr int GROUPS = RD_WARPS / WPR;
  constexpr int GLANES = WARP * WPR;
  __shared__ float red[WPR > 1 ? RD_WARPS * ROWS * B : 1];

  const int tid = threadIdx.x;
  const int warp = tid / WARP, lane = tid % WARP;
  const int group = warp / WPR, wig = warp % WPR;
  const int glane = wig * WARP + lane;
  const int nchunks = N / Chunk<T>::N;
  const uint4 *Xv = reinterpret_cast<const uint4 *>(X);

  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  if (early) {
    // Weights are not produced by any kernel, and the index list is complete (identity, or the caller's
    // promise): the first 8 KB of the first rows of this group are requested while the kernel before this
    // one is still running.
    const int m0 = blockIdx.x * GROUPS * ROWS + group * ROWS;
    constexpr int LINES = 64;
    const int row_lines = (int)min((long long)LINES, ((long long)N * (int)sizeof(T) + 127) / 128);
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
      if (m0 + j < M) {
        const long long r = load_index(idx, m0 + j, idx64);
        const char *w0 = reinterpret_cast<const char *>(W + r * ldw);
        for (int l = glane; l < row_lines; l += GLANES) prefetch_l2(w0 + (size_t)l * 128);
      }
    }
  }
  asm volatile("griddepcontrol.wait;" ::: "memory");

  const int rows_per_pass = gridDim.x * GROUPS * ROWS;
  // trip count is uniform over the block so that __syncthreads below is legal
  for (int base = blockIdx.x * GROUPS * ROWS; base < M; base += rows_per_pass) {
    const int m0 = base + group * ROWS;
    const uint4 *wp[ROWS];
    float bv[ROWS];
#pragma unroll
    for (int j = 0; j < ROWS; ++j) {
      const int m = m0 + j;
      const bool ok = m < M;
      const long long r = ok ? load_index(idx, m, idx64) : 0;
      wp[j] = reinterpret_cast<const uint4 *>(W + r * ldw);
      bv[j] = (bias != nullptr && ok) ? to_f(bias[r]) : 0.f;
      if (!ok) wp[j] = nullptr;
    }
    float acc[ROWS][B];
#pragma unroll
    for (int j = 0; j < ROWS; ++j)
#pragma unroll
      for (int b = 0; b < B; ++b) acc[j][b] = 0.f;

    for (int c0 = glane; c0 < nchunks; c0 += GLANES * U) {
      uint4 wv[ROWS][U];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = c0 + u * GLANES;
#pragma unroll
        for (int j = 0; j < ROWS; ++j) {
          if (c < nchunks && wp[j] != nullptr)
            wv[j][u] = ld_stream16(wp[j] + c);
          else
            wv[j][u] = make_uint4(0, 0, 0, 0);
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = c0 + u * GLANES;
        if (c < nchunks) {
#pragma unroll
          for (int b = 0; b < B; ++b) {
            const uint4 xv = ld_cached16(Xv + (size_t)b * nchunks + c);
#pragma unroll
            for (int j = 0; j < ROWS; ++j) acc[j][b] = dot_chunk<T>(wv[j][u], xv, acc[j][b]);
          }
        }
      }
    }
#pragma unroll
    for (int j = 0; j < ROWS; ++j)
#pragma unroll
      for (int b = 0; b < B; ++b) acc[j][b] = warp_sum(acc[j][b]);

    if (WPR > 1) {
      if (lane == 0) {
#pragma unroll
        for (int j = 0; j < ROWS; ++j)
#pragma unroll
          for (int b = 0; b < B; ++b) red[(warp * ROWS + j) * B + b] = acc[j][b];
      }
      __syncthreads();
      if (wig == 0 && lane == 0) {
#pragma unroll
        for (int j = 0; j < ROWS; ++j)
#pragma unroll
          for (int b = 0; b < B; ++b) {
            float s = 0.f;
#pragma unroll
            for (int w2 = 0; w2 < WPR; ++w2) s += red[((group * WPR + w2) * ROWS + j) * B + b];
            acc[j][b] = s;
          }
      }
    }
    if (wig == 0 && lane == 0) {
      if (is_glu(ACT)) {
        // rows 2i, 2i + 1 of the matrix are the gate and up rows of output i
#pragma unroll
        for (int j = 0; j + 1 < ROWS; j += 2) {
          const int m = m0 + j;
          if (m + 1 < M) {
#pragma unroll
            for (int b = 0; b < B; ++b)
              Y[(size_t)b * (M / 2) + m / 2] =
                  from_f<TO>(apply_glu<ACT>(acc[j][b] + bv[j], acc[j + 1][b] + bv[j + 1], act_param));
          }
        }
      } else {
#pragma unroll
        for (int j = 0; j < ROWS; ++j) {
          const int m = m0 + j;
          if (m < M) {
#pragma unroll
            for (int b = 0; b < B; ++b)
              Y[(size_t)b * M + m] = from_f<TO>(apply_act_param<ACT>(acc[j][b] + bv[j], act_param));
          }
        }
      }
    }
    if (WPR > 1) __syncthreads();  // red[] is reused by the next pass
  }
}

struct RowdotPlan {
  int wpr, rows, grid;
};

inline RowdotPlan plan_rowdot(int M, int nchunks, int B, int rows) {
  const int sms = sm_count();
  static const int k_wpr = env_int("DJV_RD_WPR", 0);  // development knobs
  static const int k_cap = env_int("DJV_RD_BLOCKS_PER_SM", 6);
  // As many warps per row as still lets every block be resident at once (4 blocks of 256 threads per SM):
  // a second, partial wave of blocks costs more than fewer lanes per row (measured: K=4096, d=9216 runs at
  // 0.77 of the HBM peak with 2 warps per row, 0.71 with 4, 0.67 with 1).
  const long long resident = (long long)sms * 4;
  int wpr = 1;
  while (wpr < 8 && (long long)ceil_div(M, (RD_WARPS / (wpr * 2)) * rows) <= resident && nchunks >= 64 * wpr * 2)
    wpr *= 2;
  if (k_wpr > 0) {
    wpr = k_wpr;
    while (wpr > 1 && nchunks < 32 * wpr) wpr /= 2;
  }
  const int groups = RD_WARPS / wpr;
  int grid = ceil_div(M, groups * rows);
  const int cap = sms * k_cap;
  if (grid > cap) grid = cap;
  if (grid < 1) grid = 1;
  return {wpr, rows, grid};
}

}  // namespace djv
