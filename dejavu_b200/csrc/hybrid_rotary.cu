// Rotary positions in place, in both pair layouts: dimension i with i + half, or 2i with 2i + 1.
#include <math.h>

#include "../../include/dejavu_b200_hybrid.h"
#include "dtype.cuh"

namespace djv {

// One block per row; the angles of the row's position are shared by its heads.
template <typename T, bool VEC, bool NEXT>  // NEXT: neighbouring dimensions form a pair
__global__ void rotary_kernel(T *__restrict__ buf, long long ld, const float *__restrict__ freqs, float amp,
                              const long long *__restrict__ pos, int n, int heads, int dim, int half) {
  extern __shared__ float cs[];  // cos[half], sin[half]
  pdl_prologue();
  const long long row = blockIdx.x;
  const int b = (int)(row / n), t = (int)(row % n);
  const float p = (float)(pos[b] + t);
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    float s, c;
    sincosf(p * freqs[i], &s, &c);
    cs[i] = c * amp;
    cs[half + i] = s * amp;
  }
  __syncthreads();
  T *x = buf + row * ld;
  if (VEC && NEXT) {  // 2 * half is a multiple of the 16-byte chunk
    constexpr int N = Chunk<T>::N;
    const int per = 2 * half / N;
    for (int k = threadIdx.x; k < heads * per; k += blockDim.x) {
      const int h = k / per, i = (k - h * per) * N;
      uint4 *pu = reinterpret_cast<uint4 *>(x + (size_t)h * dim + i);
      float u[N];
      T r[N];
      unpack_chunk<T>(*pu, u);
#pragma unroll
      for (int e = 0; e < N; e += 2) {
        const float c = cs[(i + e) / 2], s = cs[half + (i + e) / 2];
        r[e] = from_f<T>(u[e] * c - u[e + 1] * s);
        r[e + 1] = from_f<T>(u[e + 1] * c + u[e] * s);
      }
      *pu = *reinterpret_cast<uint4 *>(r);
    }
    return;
  }
  if (VEC) {  // half is a multiple of the 16-byte chunk
    constexpr int N = Chunk<T>::N;
    const int per = half / N;
    for (int k = threadIdx.x; k < heads * per; k += blockDim.x) {
      const int h = k / per, i = (k - h * per) * N;
      uint4 *pu = reinterpret_cast<uint4 *>(x + (size_t)h * dim + i);
      uint4 *pv = reinterpret_cast<uint4 *>(x + (size_t)h * dim + half + i);
      float u[N], v[N];
      T ru[N], rv[N];
      unpack_chunk<T>(*pu, u);
      unpack_chunk<T>(*pv, v);
#pragma unroll
      for (int e = 0; e < N; ++e) {
        const float c = cs[i + e], s = cs[half + i + e];
        ru[e] = from_f<T>(u[e] * c - v[e] * s);
        rv[e] = from_f<T>(v[e] * c + u[e] * s);
      }
      *pu = *reinterpret_cast<uint4 *>(ru);
      *pv = *reinterpret_cast<uint4 *>(rv);
    }
    return;
  }
  for (int k = threadIdx.x; k < heads * half; k += blockDim.x) {
    const int h = k / half, i = k % half;
    T *e = x + (size_t)h * dim + (NEXT ? 2 * i : i), *f = e + (NEXT ? 1 : half);
    const float u = to_f(*e), v = to_f(*f);
    *e = from_f<T>(u * cs[i] - v * cs[half + i]);
    *f = from_f<T>(v * cs[i] + u * cs[half + i]);
  }
}

}  // namespace djv

using namespace djv;

extern "C" int djv_rotary(int dtype, void *buf, long long ld, const float *freqs, float amp, const long long *pos, int B,
                          int n, int heads, int dim, int half, int interleaved, void *stream) {
  DJV_REQUIRE(dtype == DJV_DTYPE_BF16 || dtype == DJV_DTYPE_F32, "rotary: dtype %d", dtype);
  DJV_REQUIRE(buf && freqs && pos, "rotary: null pointer");
  DJV_REQUIRE(B >= 1 && n >= 1 && heads >= 1 && half >= 1 && 2 * half <= dim && half <= 4096 &&
                  ld >= (long long)(heads - 1) * dim + 2 * half && (long long)B * n < (1ll << 31),
              "rotary: B=%d n=%d heads=%d dim=%d half=%d", B, n, heads, dim, half);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int chunk = 16 / (int)dtype_bytes(dtype), unit = interleaved ? 2 * half : half;
  const bool vec = unit % chunk == 0 && dim % chunk == 0 && ld % chunk == 0 && aligned16(buf);
  int threads = ceil_div(vec ? heads * unit / chunk : ceil_div(heads * half, 4), WARP) * WARP;
  threads = threads > 512 ? 512 : threads;
#define DJV_ROT(T_, VEC_, NEXT_)                                                                                          \
  djv::launch_kernel(rotary_kernel<T_, VEC_, NEXT_>, B * n, threads, half * 8, st, static_cast<T_ *>(buf), ld, freqs, amp, \
                     pos, n, heads, dim, half)
#define DJV_ROT2(T_)                          \
  if (vec && interleaved) DJV_ROT(T_, true, true);       \
  else if (vec) DJV_ROT(T_, true, false);     \
  else if (interleaved) DJV_ROT(T_, false, true);        \
  else DJV_ROT(T_, false, false)
  if (dtype == DJV_DTYPE_BF16) {
    DJV_ROT2(bf16);
  } else {
    DJV_ROT2(float);
  }
#undef DJV_ROT2
#undef DJV_ROT
  count_launch();
  return check_launch("rotary");
}
