// The decode step's dense matrix products for bf16 and fp32 weights: the rowdot kernels of the sparse path with the
// identity index list, an fp32 or T result, and the epilogues of the gated MLP and of the capped logits.
#include "../../include/dejavu_b200_hybrid.h"
#include "rowdot.cuh"
#include "rowdot_mma.cuh"

namespace djv {

// Any N, any alignment: a warp per output, element by element.
template <typename T, typename TO>
__global__ void __launch_bounds__(256)
rowdot_any_kernel(TO *__restrict__ Y, const T *__restrict__ W, const T *__restrict__ X, int M, int N, long long ldw,
                  int act, float p) {
  pdl_prologue();
  const int lane = threadIdx.x % WARP, b = blockIdx.y;
  const int o = blockIdx.x * 8 + threadIdx.x / WARP;
  const int rows = is_glu(act) ? 2 : 1;
  const int M_out = M / rows;
  if (o >= M_out) return;
  float s[2] = {0.f, 0.f};
  for (int r = 0; r < rows; ++r) {
    const T *w = W + (long long)(o * rows + r) * ldw;
    for (int c = lane; c < N; c += WARP) s[r] = fmaf(to_f(w[c]), to_f(X[(size_t)b * N + c]), s[r]);
    s[r] = warp_sum(s[r]);
  }
  if (lane) return;
  float v = s[0];
  if (act == DJV_ACT_CLAMPED_GLU) v = clamped_glu(s[0], s[1], p);
  if (act == DJV_ACT_SILU_GLU) v = silu_glu(s[0], s[1]);
  if (act == DJV_ACT_SOFTCAP) v = apply_act_param<DJV_ACT_SOFTCAP>(v, p);
  Y[(size_t)b * M_out + o] = from_f<TO>(v);
}

template <typename T, typename TO, int B, int ACT>
static void launch_rowdot_dense(TO *Y, const T *W, const T *X, int M, int N, long long ldw, float param,
                                cudaStream_t st) {
  constexpr int R = (B <= 2 || is_glu(ACT)) ? 2 : 1;
  const RowdotPlan p = plan_rowdot(M, N / Chunk<T>::N, B, R);
#define DJV_RD(WPR_)                                                                                            \
  djv::launch_kernel(rowdot_kernel<T, TO, B, ACT, WPR_, R, 4>, p.grid, RD_THREADS, 0, st, Y, W, X,              \
                     static_cast<const void *>(nullptr), static_cast<const T *>(nullptr), M, N, ldw, 0, 1, param)
  switch (p.wpr) {
    case 1: DJV_RD(1); break;
    case 2: DJV_RD(2); break;
    case 4: DJV_RD(4); break;
    default: DJV_RD(8); break;
  }
#undef DJV_RD
  count_launch();
}

template <typename T, typename TO, int NT, int ACT>
static void launch_mma_dense(TO *Y, const T *W, const T *X, int B, int M, int N, long long ldw, float param,
                             cudaStream_t st) {
  static const int bps = [] {
    int n = 0;
    if (cudaOccupancyMaxActiveBlocksPerMultiprocessor(&n, rowdot_mma_kernel<T, TO, NT, ACT>, MM_THREADS, 0) !=
        cudaSuccess) {
      cudaGetLastError();
      n = 1;
    }
    return n < 1 ? 1 : n;
  }();
  const int S = rowdot_mma_split(M, N, NT, bps);
  djv::launch_kernel_cluster(rowdot_mma_kernel<T, TO, NT, ACT>, dim3(ceil_div(M, MM_ROWS), S), dim3(MM_THREADS), 0, st,
                             dim3(1, S, 1), Y, W, X, static_cast<const void *>(nullptr),
                             static_cast<const T *>(nullptr), M, N, ldw, 0, B, param);
  count_launch();
}

// tensor cores for 5 rows of x and more, 16-bit element types only
template <typename TO, int ACT>
static bool try_mma(TO *Y, const bf16 *W, const bf16 *X, int B, int M, int N, long long ldw, float param,
                    cudaStream_t st) {
  if (B < 5) return false;
  switch ((B + 7) / 8) {
    case 1: launch_mma_dense<bf16, TO, 1, ACT>(Y, W, X, B, M, N, ldw, param, st); break;
    case 2: launch_mma_dense<bf16, TO, 2, ACT>(Y, W, X, B, M, N, ldw, param, st); break;
    case 3: launch_mma_dense<bf16, TO, 3, ACT>(Y, W, X, B, M, N, ldw, param, st); break;
    default: launch_mma_dense<bf16, TO, 4, ACT>(Y, W, X, B, M, N, ldw, param, st); break;
  }
  return true;
}
template <typename TO, int ACT>
static bool try_mma(TO *, const float *, const float *, int, int, int, long long, float, cudaStream_t) {
  return false;
}

template <typename T, typename TO, int ACT>
static int dense(TO *Y, const T *W, const T *X, int B, int M, int N, long long ldw, float param, cudaStream_t st) {
  const int M_out = is_glu(ACT) ? M / 2 : M;
  if (N % Chunk<T>::N != 0 || ldw % Chunk<T>::N != 0 || !aligned16(W) || !aligned16(X)) {
    djv::launch_kernel(rowdot_any_kernel<T, TO>, dim3(ceil_div(M_out, 8), B), dim3(256), 0, st, Y, W, X, M, N, ldw, ACT,
                       param);
    count_launch();
    return DJV_OK;
  }
  if (try_mma<TO, ACT>(Y, W, X, B, M, N, ldw, param, st)) return DJV_OK;
  for (int b0 = 0; b0 < B; b0 += 4) {
    TO *y = Y + (size_t)b0 * M_out;
    const T *x = X + (size_t)b0 * N;
    switch (B - b0) {
      case 1: launch_rowdot_dense<T, TO, 1, ACT>(y, W, x, M, N, ldw, param, st); break;
      case 2: launch_rowdot_dense<T, TO, 2, ACT>(y, W, x, M, N, ldw, param, st); break;
      case 3: launch_rowdot_dense<T, TO, 3, ACT>(y, W, x, M, N, ldw, param, st); break;
      default: launch_rowdot_dense<T, TO, 4, ACT>(y, W, x, M, N, ldw, param, st); break;
    }
  }
  return DJV_OK;
}

}  // namespace djv

using namespace djv;

extern "C" int djv_dense_gemv(int dtype, int out_dtype, void *y, const void *w, const void *x, int B, int N, int M,
                              long long ldw, int act, float act_param, void *stream) {
  DJV_REQUIRE(y && w && x, "dense_gemv: null pointer");
  DJV_REQUIRE(dtype == DJV_DTYPE_BF16 || dtype == DJV_DTYPE_F32, "dense_gemv: dtype %d", dtype);
  DJV_REQUIRE(out_dtype == dtype || out_dtype == DJV_DTYPE_F32, "dense_gemv: output type %d", out_dtype);
  DJV_REQUIRE(B >= 1 && B <= DJV_MAX_BATCH, "dense_gemv: batch %d outside [1,%d]", B, DJV_MAX_BATCH);
  DJV_REQUIRE(N >= 1 && M >= 1 && ldw >= N, "dense_gemv: N=%d M=%d ldw=%lld", N, M, ldw);
  DJV_REQUIRE(!is_glu(act) || M % 2 == 0, "dense_gemv: a gated unit needs an even number of rows");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  int rc = DJV_OK;
#define DJV_DENSE(T_, TO_, ACT_)                                                                                   \
  rc = dense<T_, TO_, ACT_>(static_cast<TO_ *>(y), static_cast<const T_ *>(w), static_cast<const T_ *>(x), B, M, N, \
                            ldw, act_param, st)
  const bool b16 = dtype == DJV_DTYPE_BF16, f32_out = out_dtype == DJV_DTYPE_F32;
  if (act == DJV_ACT_ID) {
    if (b16 && !f32_out) DJV_DENSE(bf16, bf16, DJV_ACT_ID);
    else if (b16) DJV_DENSE(bf16, float, DJV_ACT_ID);
    else DJV_DENSE(float, float, DJV_ACT_ID);
  } else if (act == DJV_ACT_SOFTCAP && f32_out) {
    if (b16) DJV_DENSE(bf16, float, DJV_ACT_SOFTCAP);
    else DJV_DENSE(float, float, DJV_ACT_SOFTCAP);
  } else if (act == DJV_ACT_CLAMPED_GLU && out_dtype == dtype) {
    if (b16) DJV_DENSE(bf16, bf16, DJV_ACT_CLAMPED_GLU);
    else DJV_DENSE(float, float, DJV_ACT_CLAMPED_GLU);
  } else if (act == DJV_ACT_SILU_GLU && out_dtype == dtype) {
    if (b16) DJV_DENSE(bf16, bf16, DJV_ACT_SILU_GLU);
    else DJV_DENSE(float, float, DJV_ACT_SILU_GLU);
  } else {
    set_error("dense_gemv: activation %d with output type %d is not compiled", act, out_dtype);
    return DJV_ERR_UNSUPPORTED;
  }
#undef DJV_DENSE
  if (rc) return rc;
  return check_launch("dense_gemv");
}
