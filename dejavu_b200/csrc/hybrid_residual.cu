// The boundary between two sublayers of a decoder with hyper-connected residual streams: stream update from the
// previous sublayer's output, weighted sum of the streams, RMS norm. One block per row; every stream element is read
// and written once. Bytes per row: S*D*4 read + S*D*4 written + D*4 (y) + D*sizeof(T) (h).
// Also the boundary of a decoder with one stream and norms on both sides of a sublayer, and the two small elementwise
// kernels of the prompt pass (gated units, logit softcap).
#include "../../include/dejavu_b200_hybrid.h"
#include "dtype.cuh"
#include "rowdot.cuh"

namespace djv {

constexpr int HS_THREADS = 512;

struct HyperArgs {
  void *h;
  float *x_out;
  const float *x_in, *y, *mix, *w_out, *w_in, *gamma;
  float eps;
  const int *row_list;
  const long long *ids;
  const void *embed;
  int D, vocab;
};

template <typename T, int S, int V>  // V columns at a time: 4 (16-byte accesses) or 1
__global__ void __launch_bounds__(HS_THREADS) hyper_step_kernel(HyperArgs a) {
  extern __shared__ float u_s[];  // D
  __shared__ float coef[S * S + 2 * S];
  __shared__ float red[HS_THREADS / WARP];
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  const int tid = threadIdx.x;
  // the coefficients are weights: no kernel of the step writes them
  if (tid < S * S) coef[tid] = a.y ? a.mix[tid] : (tid / S == tid % S ? 1.f : 0.f);
  if (tid >= 64 && tid < 64 + S) coef[S * S + tid - 64] = a.y ? a.w_out[tid - 64] : 0.f;
  if (tid >= 96 && tid < 96 + S) coef[S * S + S + tid - 96] = a.w_in ? a.w_in[tid - 96] : 1.f;
  asm volatile("griddepcontrol.wait;" ::: "memory");
  __syncthreads();
  const int D = a.D;
  const int row = a.row_list ? a.row_list[blockIdx.x] : blockIdx.x;
  const float *x = a.x_in ? a.x_in + (size_t)row * S * D : nullptr;
  const T *e = nullptr;
  if (!a.x_in) {
    const long long id = a.ids[row];
    e = static_cast<const T *>(a.embed) + (size_t)(id < 0 ? 0 : (id >= a.vocab ? a.vocab - 1 : id)) * D;
  }
  float ss = 0.f;
#pragma unroll 2
  for (int c = tid * V; c < D; c += blockDim.x * V) {
    float xs[S][V], yv[V], u[V];
    if (x) {
#pragma unroll
      for (int s = 0; s < S; ++s) {
        if (V == 4) {
          const float4 t = *reinterpret_cast<const float4 *>(x + (size_t)s * D + c);
          xs[s][0] = t.x; xs[s][1 % V] = t.y; xs[s][2 % V] = t.z; xs[s][3 % V] = t.w;
        } else {
          xs[s][0] = x[(size_t)s * D + c];
        }
      }
    } else {
#pragma unroll
      for (int v = 0; v < V; ++v) {
        const float t = to_f(e[c + v]);
#pragma unroll
        for (int s = 0; s < S; ++s) xs[s][v] = t;
      }
    }
#pragma unroll
    for (int v = 0; v < V; ++v) yv[v] = u[v] = 0.f;
    if (a.y) {
      if (V == 4) {
        const float4 t = *reinterpret_cast<const float4 *>(a.y + (size_t)row * D + c);
        yv[0] = t.x; yv[1 % V] = t.y; yv[2 % V] = t.z; yv[3 % V] = t.w;
      } else {
        yv[0] = a.y[(size_t)row * D + c];
      }
    }
#pragma unroll
    for (int t = 0; t < S; ++t) {
      float nv[V];
#pragma unroll
      for (int v = 0; v < V; ++v) {
        float acc = coef[S * S + t] * yv[v];
#pragma unroll
        for (int s = 0; s < S; ++s) acc = fmaf(coef[s * S + t], xs[s][v], acc);
        nv[v] = acc;
        u[v] = fmaf(coef[S * S + S + t], acc, u[v]);
      }
      if (a.x_out) {
        float *dst = a.x_out + ((size_t)row * S + t) * D + c;
        if (V == 4)
          *reinterpret_cast<float4 *>(dst) = make_float4(nv[0], nv[1 % V], nv[2 % V], nv[3 % V]);
        else
          dst[0] = nv[0];
      }
    }
#pragma unroll
    for (int v = 0; v < V; ++v) {
      u_s[c + v] = u[v];
      ss = fmaf(u[v], u[v], ss);
    }
  }
  if (!a.gamma) return;
  ss = warp_sum(ss);
  if (tid % WARP == 0) red[tid / WARP] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int w = 0; w < blockDim.x / WARP; ++w) tot += red[w];
  const float rstd = 1.f / sqrtf(tot / (float)D + a.eps);
  T *h = static_cast<T *>(a.h) + (size_t)blockIdx.x * D;
  for (int c = tid * V; c < D; c += blockDim.x * V) {  // the same columns this thread wrote into u_s
    T o[V];
#pragma unroll
    for (int v = 0; v < V; ++v) o[v] = from_f<T>(u_s[c + v] * rstd * a.gamma[c + v]);
    if (V == 4 && sizeof(T) == 2)
      *reinterpret_cast<uint2 *>(h + c) = *reinterpret_cast<uint2 *>(o);
    else if (V == 4)
      *reinterpret_cast<uint4 *>(h + c) = *reinterpret_cast<uint4 *>(o);
    else
      h[c] = o[0];
  }
}

template <typename T, int V>
static int launch_hyper(const HyperArgs &a, int R, int S, cudaStream_t st) {
  int threads = ceil_div(ceil_div(a.D, V), WARP) * WARP;
  // many rows: smaller blocks, so that the multiprocessor always has one that streams while others reduce and store
  // (measured at 4096 rows of 4 streams: 0.92 of the copy peak with 256 threads, 0.75 with 512); few rows: wide blocks
  const int most = R > 2 * sm_count() ? HS_THREADS / 2 : HS_THREADS;
  if (threads > most) threads = most;
  if (threads < 128) threads = 128;
  const size_t smem = (size_t)a.D * 4;
#define DJV_HS(S_)                                                                                      \
  case S_:                                                                                              \
    if (smem > 48 * 1024)                                                                               \
      cudaFuncSetAttribute(hyper_step_kernel<T, S_, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    djv::launch_kernel(hyper_step_kernel<T, S_, V>, R, threads, smem, st, a);                           \
    break
  switch (S) {
    DJV_HS(1);
    DJV_HS(2);
    DJV_HS(3);
    DJV_HS(4);
    DJV_HS(5);
    DJV_HS(6);
    DJV_HS(7);
    DJV_HS(8);
  }
#undef DJV_HS
  count_launch();
  return check_launch("hyper_step");
}

// ---- one stream, norms on both sides -------------------------------------------------------------------------------
//   s = y + sum of the row's parts;  new = x + (norm of) s;  h = norm of new
// A norm's weight is base + gamma. One block per row, the row stays in registers (NI * 4 columns per thread) between the
// two sums of squares. Bytes per row: D*4 read + D*4 written + D*4 (y) or parts + D*sizeof(T) (h).
struct ResidualArgs {
  void *h;
  float *x_out;
  const float *x_in, *y;
  const void *parts;
  const int *part_rows;
  int n_parts;
  const float *gamma_y, *gamma;
  float base, eps;
  const int *row_list;
  const long long *ids;
  const void *embed;
  int D, vocab;
};

__device__ __forceinline__ float block_sum(float v, float *red) {
  v = warp_sum(v);
  if (threadIdx.x % WARP == 0) red[threadIdx.x / WARP] = v;
  __syncthreads();
  float s = 0.f;
  for (int w = 0; w < (int)blockDim.x / WARP; ++w) s += red[w];
  return s;
}

template <typename T>
__device__ __forceinline__ void load4(const T *p, float (&v)[4]) {
  if (sizeof(T) == 4) {
    const float4 t = *reinterpret_cast<const float4 *>(p);
    v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
  } else {
    const uint2 t = *reinterpret_cast<const uint2 *>(p);
    const float2 a = b2f(t.x), b = b2f(t.y);
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
  }
}

template <typename T, int NI>  // D <= NI * 4 * blockDim.x, 16-byte accesses; NI == 0: any D, the row in shared memory
__global__ void __launch_bounds__(512) residual_step_kernel(ResidualArgs a) {
  extern __shared__ float sm[];  // NI == 0: [D] sums, [D] new values
  __shared__ float red[2][32];
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  const int tid = threadIdx.x, D = a.D;
  constexpr int W = NI > 0 ? NI : 1;
  float gy[W][4], gh[W][4];  // norm weights: no kernel of the step writes them
  if constexpr (NI > 0 && NI <= 2) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = (i * blockDim.x + tid) * 4;
      if (c < D && a.gamma_y) load4(a.gamma_y + c, gy[i]);
      if (c < D && a.gamma) load4(a.gamma + c, gh[i]);
    }
  }
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const int row = a.row_list ? a.row_list[blockIdx.x] : blockIdx.x;
  const float *x = a.x_in ? a.x_in + (size_t)row * D : nullptr, *y = a.y ? a.y + (size_t)row * D : nullptr;
  const T *e = nullptr, *parts = static_cast<const T *>(a.parts);
  if (!x) {
    const long long id = a.ids[row];
    e = static_cast<const T *>(a.embed) + (size_t)(id < 0 ? 0 : (id >= a.vocab ? a.vocab - 1 : id)) * D;
  }
  const int *pr = a.part_rows + (size_t)row * a.n_parts;
  const int np = parts ? a.n_parts : 0;
  T *h = static_cast<T *>(a.h) + (size_t)blockIdx.x * D;
  float ss = 0.f;
  if constexpr (NI > 0) {
    float xv[NI][4], yv[NI][4];
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = (i * blockDim.x + tid) * 4;
#pragma unroll
      for (int v = 0; v < 4; ++v) xv[i][v] = yv[i][v] = 0.f;
      if (c < D) {
        if (x) load4(x + c, xv[i]);
        else load4(e + c, xv[i]);
        if (y) load4(y + c, yv[i]);
      }
    }
    for (int k = 0; k < np; ++k) {
      const T *p = parts + (size_t)pr[k] * D;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int c = (i * blockDim.x + tid) * 4;
        float t[4] = {0.f, 0.f, 0.f, 0.f};
        if (c < D) load4(p + c, t);
#pragma unroll
        for (int v = 0; v < 4; ++v) yv[i][v] += t[v];
      }
    }
    float r = 1.f;
    if (a.gamma_y) {
#pragma unroll
      for (int i = 0; i < NI; ++i)
#pragma unroll
        for (int v = 0; v < 4; ++v) ss = fmaf(yv[i][v], yv[i][v], ss);
      r = 1.f / sqrtf(block_sum(ss, red[0]) / (float)D + a.eps);
    }
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = (i * blockDim.x + tid) * 4;
      if (c >= D) continue;
      if (NI > 2 && a.gamma_y) load4(a.gamma_y + c, gy[i]);
#pragma unroll
      for (int v = 0; v < 4; ++v) {
        xv[i][v] += a.gamma_y ? yv[i][v] * r * (a.base + gy[i][v]) : yv[i][v];
        ss = fmaf(xv[i][v], xv[i][v], ss);
      }
      if (a.x_out)
        *reinterpret_cast<float4 *>(a.x_out + (size_t)row * D + c) = make_float4(xv[i][0], xv[i][1], xv[i][2], xv[i][3]);
    }
    if (!a.gamma) return;
    r = 1.f / sqrtf(block_sum(ss, red[1]) / (float)D + a.eps);
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int c = (i * blockDim.x + tid) * 4;
      if (c >= D) continue;
      if (NI > 2) load4(a.gamma + c, gh[i]);
      T o[4];
#pragma unroll
      for (int v = 0; v < 4; ++v) o[v] = from_f<T>(xv[i][v] * r * (a.base + gh[i][v]));
      if (sizeof(T) == 2) *reinterpret_cast<uint2 *>(h + c) = *reinterpret_cast<uint2 *>(o);
      else *reinterpret_cast<uint4 *>(h + c) = *reinterpret_cast<uint4 *>(o);
    }
  } else {
    float *ys = sm, *xs = sm + D;
    for (int c = tid; c < D; c += blockDim.x) {  // (every thread comes back to its own columns)
      float v = y ? y[c] : 0.f;
      for (int k = 0; k < np; ++k) v += to_f(parts[(size_t)pr[k] * D + c]);
      ys[c] = v;
      ss = fmaf(v, v, ss);
    }
    const float r = a.gamma_y ? 1.f / sqrtf(block_sum(ss, red[0]) / (float)D + a.eps) : 1.f;
    ss = 0.f;
    for (int c = tid; c < D; c += blockDim.x) {
      const float v = (x ? x[c] : to_f(e[c])) + ys[c] * r * (a.gamma_y ? a.base + a.gamma_y[c] : 1.f);
      xs[c] = v;
      ss = fmaf(v, v, ss);
      if (a.x_out) a.x_out[(size_t)row * D + c] = v;
    }
    if (!a.gamma) return;
    const float rh = 1.f / sqrtf(block_sum(ss, red[1]) / (float)D + a.eps);
    for (int c = tid; c < D; c += blockDim.x) h[c] = from_f<T>(xs[c] * rh * (a.base + a.gamma[c]));
  }
}

template <typename T>
static int launch_residual(const ResidualArgs &a, int R, bool vec, cudaStream_t st) {
  const int groups = ceil_div(a.D, 4);  // groups of 4 columns
  // many rows: fewer threads with more columns each, so that a multiprocessor streams several rows at once
  int threads = R > 2 * sm_count() ? 256 : 512;
  while (threads > 64 && threads / 2 >= groups) threads /= 2;
  if (groups > 4 * threads) threads = 512;
  const int ni = ceil_div(groups, threads);
#define DJV_GO(NI_, SM_)                                                                                                 \
  {                                                                                                                      \
    if ((SM_) > 48 * 1024)                                                                                               \
      cudaFuncSetAttribute(residual_step_kernel<T, NI_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)(SM_));       \
    djv::launch_kernel(residual_step_kernel<T, NI_>, R, threads, SM_, st, a);                                            \
  }
  if (vec && ni == 1) DJV_GO(1, 0)
  else if (vec && ni == 2) DJV_GO(2, 0)
  else if (vec && ni <= 4) DJV_GO(4, 0)
  else DJV_GO(0, (size_t)a.D * 8)
#undef DJV_GO
  count_launch();
  return check_launch("residual_step");
}

template <typename T, int ACT>
__global__ void glu_kernel(T *__restrict__ y, const T *__restrict__ gu, long long total, float limit) {
  pdl_prologue();
  // two groups of 4 outputs per thread, a block apart: both loads in flight
  const long long g0 = (long long)blockIdx.x * blockDim.x * 8 + threadIdx.x * 4;
  uint4 v[2];
  bool wide[2];
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const long long i0 = g0 + (long long)k * blockDim.x * 4;
    wide[k] = sizeof(T) == 2 && total - i0 >= 4;
    if (wide[k]) v[k] = ld_stream16(gu + i0 * 2);
  }
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const long long i0 = g0 + (long long)k * blockDim.x * 4;
    if (wide[k]) {
      float f[8];
      unpack_chunk<bf16>(v[k], f);
      uint2 o;
      o.x = pack_bf16(apply_glu<ACT>(f[0], f[1], limit), apply_glu<ACT>(f[2], f[3], limit));
      o.y = pack_bf16(apply_glu<ACT>(f[4], f[5], limit), apply_glu<ACT>(f[6], f[7], limit));
      *reinterpret_cast<uint2 *>(y + i0) = o;
    } else {
      for (long long i = i0; i < total && i < i0 + 4; ++i)
        y[i] = from_f<T>(apply_glu<ACT>(to_f(gu[2 * i]), to_f(gu[2 * i + 1]), limit));
    }
  }
}

__global__ void softcap_kernel(float *y, long long n, float cap) {
  pdl_prologue();
  const long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) y[i] = cap * tanhf(y[i] / cap);
}

}  // namespace djv

using namespace djv;

extern "C" int djv_hyper_step(int dtype, void *h, float *x_out, const float *x_in, const float *y, const float *mix,
                              const float *w_out, const float *w_in, const float *gamma, float eps,
                              const int32_t *row_list, const long long *ids, const void *embed, int R, int S, int D,
                              int vocab, void *stream) {
  DJV_REQUIRE(dtype == DJV_DTYPE_BF16 || dtype == DJV_DTYPE_F32, "hyper_step: dtype %d", dtype);
  DJV_REQUIRE(x_in || (ids && embed && vocab > 0), "hyper_step: neither streams nor an embedding given");
  DJV_REQUIRE(!y || (mix && w_out), "hyper_step: y without mix and out coefficients");
  DJV_REQUIRE(!gamma || h || R == 0, "hyper_step: null output");
  DJV_REQUIRE(S >= 1 && S <= 8, "hyper_step: %d streams (1..8 are supported)", S);
  DJV_REQUIRE(D >= 1 && D <= 49152 && R >= 0, "hyper_step: D=%d R=%d", D, R);
  if (R == 0) return DJV_OK;
  const HyperArgs a{h, x_out, x_in, y, mix, w_out, w_in, gamma, eps, row_list, ids, embed, D, vocab};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool vec = D % 4 == 0 && aligned16(x_in) && aligned16(x_out) && aligned16(y) && aligned16(h);
  if (dtype == DJV_DTYPE_BF16) return vec ? launch_hyper<bf16, 4>(a, R, S, st) : launch_hyper<bf16, 1>(a, R, S, st);
  return vec ? launch_hyper<float, 4>(a, R, S, st) : launch_hyper<float, 1>(a, R, S, st);
}

extern "C" int djv_residual_step(int dtype, void *h, float *x_out, const float *x_in, const float *y, const void *parts,
                                 const int32_t *part_rows, int n_parts, const float *gamma_y, const float *gamma,
                                 float base, float eps, const int32_t *row_list, const long long *ids, const void *embed,
                                 int R, int D, int vocab, void *stream) {
  DJV_REQUIRE(dtype == DJV_DTYPE_BF16 || dtype == DJV_DTYPE_F32, "residual_step: dtype %d", dtype);
  DJV_REQUIRE(x_in || (ids && embed && vocab > 0), "residual_step: neither a residual nor an embedding given");
  DJV_REQUIRE(!parts || (part_rows && n_parts >= 1), "residual_step: parts without their rows");
  DJV_REQUIRE(!gamma || h || R == 0, "residual_step: null output");
  DJV_REQUIRE(D >= 1 && D <= 24576 && R >= 0, "residual_step: D=%d R=%d", D, R);
  if (R == 0) return DJV_OK;
  const ResidualArgs a{h,    x_out, x_in, y,        parts, part_rows, n_parts, gamma_y, gamma,
                       base, eps,   row_list, ids, embed, D,         vocab};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool vec = D % 4 == 0 && aligned16(x_in) && aligned16(x_out) && aligned16(y) && aligned16(h) && aligned16(parts) &&
                   aligned16(gamma_y) && aligned16(gamma) && aligned16(embed);
  return dtype == DJV_DTYPE_BF16 ? launch_residual<bf16>(a, R, vec, st) : launch_residual<float>(a, R, vec, st);
}

extern "C" int djv_glu(int dtype, void *y, const void *gu, long long R, int F, int act, float limit, void *stream) {
  DJV_REQUIRE(dtype == DJV_DTYPE_BF16 || dtype == DJV_DTYPE_F32, "glu: dtype %d", dtype);
  DJV_REQUIRE(y && gu && aligned16(y) && aligned16(gu), "glu: null or misaligned pointer");
  DJV_REQUIRE(R >= 0 && F >= 1 && is_glu(act) && limit >= 0.f, "glu: R=%lld F=%d act=%d limit=%g", R, F, act, (double)limit);
  const long long total = R * F;
  if (total == 0) return DJV_OK;
  const long long blocks = (total + 2047) / 2048;
  DJV_REQUIRE(blocks < (1ll << 31), "glu: too many elements");
  cudaStream_t st = static_cast<cudaStream_t>(stream);
#define DJV_GLU(T_, ACT_)                                                                             \
  djv::launch_kernel(glu_kernel<T_, ACT_>, (unsigned)blocks, 256, 0, st, static_cast<T_ *>(y),        \
                     static_cast<const T_ *>(gu), total, limit)
  if (dtype == DJV_DTYPE_BF16) {
    if (act == DJV_ACT_CLAMPED_GLU) DJV_GLU(bf16, DJV_ACT_CLAMPED_GLU);
    else DJV_GLU(bf16, DJV_ACT_SILU_GLU);
  } else {
    if (act == DJV_ACT_CLAMPED_GLU) DJV_GLU(float, DJV_ACT_CLAMPED_GLU);
    else DJV_GLU(float, DJV_ACT_SILU_GLU);
  }
#undef DJV_GLU
  count_launch();
  return check_launch("glu");
}

extern "C" int djv_softcap(float *y, long long n, float cap, void *stream) {
  DJV_REQUIRE(y && n >= 0 && cap > 0.f, "softcap: null pointer, n=%lld or cap=%g", n, (double)cap);
  if (n == 0) return DJV_OK;
  DJV_REQUIRE((n + 255) / 256 < (1ll << 31), "softcap: too many elements");
  djv::launch_kernel(softcap_kernel, (unsigned)((n + 255) / 256), 256, 0, static_cast<cudaStream_t>(stream), y, n, cap);
  count_launch();
  return check_launch("softcap");
}
