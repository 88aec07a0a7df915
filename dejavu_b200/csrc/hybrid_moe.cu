// Routed feed-forward: every token goes through the `top` experts with the largest router scores sigmoid(z); an expert is a
// gated unit whose input is the token's activation times its score.
//
// A prompt portion is sorted by expert on the device (no host synchronisation) and runs as grouped matrix products: this
// file has the sorting and a CUDA-core form of the product for any size, hybrid_moe_gemm.cu the tensor-core form. A decode
// step runs two kernels on the chosen experts' weights, each weight row read once per sequence that uses it; a shared
// expert, which every token uses, can run in the same two kernels.
#include "../../include/dejavu_b200_routed.h"
#include "hybrid_moe.cuh"

namespace djv {

constexpr int MAX_TOP = 16, MAX_EXPERTS = 1024;

// The `top` largest of z[0 .. E) by one warp, ties to the lower index. Lane k < top returns (index, value) of place k.
__device__ __forceinline__ void warp_topk(const float *z, int E, int top, int &index, float &value) {
  const int lane = threadIdx.x % WARP;
  float last = INFINITY;  // the choice before, and its index: what comes after it in the order (value down, index up)
  int last_i = -1;
  index = 0;
  value = 0.f;
  for (int k = 0; k < top; ++k) {
    float best = -INFINITY;
    int at = 0x7fffffff;
    for (int e = lane; e < E; e += WARP) {
      const float v = z[e];
      const bool open = v < last || (v == last && e > last_i);
      if (open && (v > best || at == 0x7fffffff)) {
        best = v;
        at = e;
      }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
      const float ov = __shfl_xor_sync(0xffffffffu, best, o);
      const int oi = __shfl_xor_sync(0xffffffffu, at, o);
      if (oi != 0x7fffffff && (at == 0x7fffffff || ov > best || (ov == best && oi < at))) {
        best = ov;
        at = oi;
      }
    }
    last = best;
    last_i = at;
    if (lane == k) {
      index = at < E ? at : 0;  // (a row that is not a number chooses something inside the range)
      value = best;
    }
  }
}

// ---- prompt portions: sorting ------------------------------------------------------------------------------------
constexpr int RT_WARPS = 8, RT_TOKENS = 64;

// choices of every token, and each choice's place among its expert's rows
__global__ void __launch_bounds__(RT_WARPS * WARP) moe_route_kernel(const float *__restrict__ z, int n, int E, int top,
                                                                    int *__restrict__ expert, int *__restrict__ place,
                                                                    float *__restrict__ weight, int *__restrict__ count) {
  extern __shared__ int sm[];
  int *cnt = sm, *base = cnt + E, *pick = base + E, *own = pick + RT_TOKENS * top;  // [E], [E], [tokens][top] x2
  pdl_prologue();
  const int tid = threadIdx.x, warp = tid / WARP, lane = tid % WARP;
  const int t0 = blockIdx.x * RT_TOKENS, tn = min(RT_TOKENS, n - t0);
  for (int e = tid; e < E; e += blockDim.x) cnt[e] = 0;
  __syncthreads();
  for (int t = warp; t < tn; t += RT_WARPS) {
    int e;
    float v;
    warp_topk(z + (size_t)(t0 + t) * E, E, top, e, v);
    if (lane < top) {
      pick[t * top + lane] = e;
      own[t * top + lane] = atomicAdd(cnt + e, 1);
      weight[(size_t)(t0 + t) * top + lane] = sigmoid_f(v);
    }
  }
  __syncthreads();
  for (int e = tid; e < E; e += blockDim.x) base[e] = cnt[e] ? atomicAdd(count + e, cnt[e]) : 0;
  __syncthreads();
  for (int i = tid; i < tn * top; i += blockDim.x) {
    expert[(size_t)t0 * top + i] = pick[i];
    place[(size_t)t0 * top + i] = base[pick[i]] + own[i];
  }
}

// rows in the order of their experts: copies of the activations, weights, and where each choice went (over `place`)
template <typename T, bool VEC>
__global__ void __launch_bounds__(256) moe_scatter_kernel(T *__restrict__ xs, const T *__restrict__ x,
                                                          const int *__restrict__ expert, int *__restrict__ place,
                                                          const float *__restrict__ weight, float *__restrict__ ws,
                                                          const int *__restrict__ count, int *__restrict__ offsets, int n,
                                                          int E, int top, int D) {
  extern __shared__ int off[];  // E + 1
  pdl_prologue();
  const int tid = threadIdx.x, lane = tid % WARP;
  if (tid < WARP) {
    int run = 0;
    for (int e0 = 0; e0 < E; e0 += WARP) {
      const int c = e0 + lane < E ? count[e0 + lane] : 0;
      int s = c;
#pragma unroll
      for (int o = 1; o < WARP; o <<= 1) {
        const int up = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s += up;
      }
      if (e0 + lane < E) off[e0 + lane] = run + s - c;
      run += __shfl_sync(0xffffffffu, s, WARP - 1);
    }
    if (lane == 0) off[E] = run;
  }
  __syncthreads();
  if (blockIdx.x == 0)
    for (int e = tid; e <= E; e += blockDim.x) offsets[e] = off[e];
  for (int i = blockIdx.x; i < n * top; i += gridDim.x) {
    const int to = off[expert[i]] + place[i];
    __syncthreads();  // everybody has read place[i]
    if (tid == 0) {
      place[i] = to;
      ws[to] = weight[i];
    }
    const T *src = x + (size_t)(i / top) * D;
    T *dst = xs + (size_t)to * D;
    if (VEC) {
      constexpr int N = Chunk<T>::N;
      for (int c = tid; c < D / N; c += blockDim.x)
        reinterpret_cast<uint4 *>(dst)[c] = reinterpret_cast<const uint4 *>(src)[c];
    } else {
      for (int c = tid; c < D; c += blockDim.x) dst[c] = src[c];
    }
  }
}

// ---- prompt portions: grouped product on the CUDA cores ------------------------------------------------------------
constexpr int GG_M = 64, GG_N = 64, GG_K = 16, GG_THREADS = 256;

template <typename T>
__global__ void __launch_bounds__(GG_THREADS) moe_grouped_kernel(GroupedArgs a) {
  __shared__ float xs[GG_K][GG_M + 4], wsm[GG_K][GG_N + 4];
  __shared__ int found[4];
  pdl_prologue();
  const int tid = threadIdx.x;
  if (tid == 0) {
    int e, r0, r1;
    found[0] = grouped_tile(a.offsets, a.E, GG_M, blockIdx.y, e, r0, r1);
    found[1] = e;
    found[2] = r0;
    found[3] = r1;
  }
  __syncthreads();
  if (!found[0]) return;
  const int e = found[1], r0 = found[2], rows = min(GG_M, found[3] - r0), n0 = blockIdx.x * GG_N;
  const T *x = static_cast<const T *>(a.x) + (size_t)r0 * a.K;
  const T *w = static_cast<const T *>(a.w) + ((size_t)e * a.N + n0) * a.K;
  const int tm = tid / 16 * 4, tn = tid % 16 * 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < a.K; k0 += GG_K) {
    for (int i = tid; i < GG_M * GG_K; i += GG_THREADS) {
      const int r = i / GG_K, k = i % GG_K;
      xs[k][r] = r < rows && k0 + k < a.K ? to_f(x[(size_t)r * a.K + k0 + k]) : 0.f;
      wsm[k][r] = n0 + r < a.N && k0 + k < a.K ? to_f(w[(size_t)r * a.K + k0 + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < GG_K; ++k) {
      float u[4], v[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        u[i] = xs[k][tm + i];
        v[i] = wsm[k][tn + i];
      }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(u[i], v[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    if (tm + i >= rows) continue;
    const size_t r = (size_t)r0 + tm + i;
    const float s = a.scale ? a.scale[r] : 1.f;
    if (a.glu) {
#pragma unroll
      for (int j = 0; j < 4; j += 2)
        if (n0 + tn + j + 1 < a.N)
          static_cast<T *>(a.y)[r * (a.N / 2) + (n0 + tn + j) / 2] = from_f<T>(silu_glu(s * acc[i][j], s * acc[i][j + 1]));
    } else {
#pragma unroll
      for (int j = 0; j < 4; ++j)
        if (n0 + tn + j < a.N) static_cast<T *>(a.y)[r * a.N + n0 + tn + j] = from_f<T>(s * acc[i][j]);
    }
  }
}

// ---- decode ----------------------------------------------------------------------------------------------------
struct MoeDecodeArgs {
  float *y;               // (B, D)
  void *act;              // (B, slots, ld_act): slot k < top is a token's k-th expert, slot top the shared one
  int *chosen;            // (B, top)
  const void *x;          // (B, D)
  const float *z;         // (B, E)
  const void *w_gu, *w_down;        // (E, 2F, D), (E, D, F)
  const void *shared_gu, *shared_down;  // (2F', D), (D, F'), or null
  const float *init;      // (B, D) added to y, or null
  int B, E, top, D, F, F_shared, ld_act;
};

constexpr int MO_THREADS = 256, MO_WARPS = MO_THREADS / WARP;

// dot products of R rows of w (stride ld) with x, N elements, by a warp: U 16-byte chunks per lane and row in flight
template <typename T, bool VEC, int R, int U>
__device__ __forceinline__ void warp_rows(const T *w, size_t ld, const T *x, int n, float (&acc)[R]) {
  const int lane = threadIdx.x % WARP;
  if (VEC) {
    const int nch = n / Chunk<T>::N;
    for (int c0 = lane; c0 < nch; c0 += WARP * U) {
      uint4 v[R][U];
#pragma unroll
      for (int u = 0; u < U; ++u)
#pragma unroll
        for (int r = 0; r < R; ++r) {
          const int c = c0 + u * WARP;
          v[r][u] = c < nch ? ld_stream16(reinterpret_cast<const uint4 *>(w + r * ld) + c) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = c0 + u * WARP;
        if (c < nch) {
          const uint4 xv = *(reinterpret_cast<const uint4 *>(x) + c);
#pragma unroll
          for (int r = 0; r < R; ++r) acc[r] = dot_chunk<T>(v[r][u], xv, acc[r]);
        }
      }
    }
  } else {
    for (int c = lane; c < n; c += WARP)
#pragma unroll
      for (int r = 0; r < R; ++r) acc[r] = fmaf(to_f(w[r * ld + c]), to_f(x[c]), acc[r]);
  }
}

// grid (B, tiles of outputs, slots): sequences that use the same weights run side by side
template <typename T, bool VEC>
__global__ void __launch_bounds__(MO_THREADS) moe_decode_up_kernel(MoeDecodeArgs a) {
  __shared__ int pick_s;
  __shared__ float weight_s;
  pdl_prologue();
  const int b = blockIdx.x, slot = blockIdx.z, lane = threadIdx.x % WARP, warp = threadIdx.x / WARP;
  const bool shared = slot == a.top;
  const int F = shared ? a.F_shared : a.F, o = blockIdx.y * MO_WARPS + warp;
  if ((int)blockIdx.y * MO_WARPS >= F) return;
  if (!shared) {
    if (warp == 0) {
      int e;
      float v;
      warp_topk(a.z + (size_t)b * a.E, a.E, slot + 1, e, v);
      if (lane == slot) {
        pick_s = e;
        weight_s = sigmoid_f(v);
        if (blockIdx.y == 0) a.chosen[b * a.top + slot] = e;
      }
    }
    __syncthreads();
  }
  if (o >= F) return;
  const float wt = shared ? 1.f : weight_s;
  const T *w = shared ? static_cast<const T *>(a.shared_gu) : static_cast<const T *>(a.w_gu) + (size_t)pick_s * 2 * a.F * a.D;
  float acc[2] = {0.f, 0.f};
  warp_rows<T, VEC, 2, 4>(w + (size_t)2 * o * a.D, a.D, static_cast<const T *>(a.x) + (size_t)b * a.D, a.D, acc);
  acc[0] = warp_sum(acc[0]);
  acc[1] = warp_sum(acc[1]);
  if (lane == 0)
    static_cast<T *>(a.act)[((size_t)b * gridDim.z + slot) * a.ld_act + o] = from_f<T>(silu_glu(wt * acc[0], wt * acc[1]));
}

template <typename T, bool VEC>
__global__ void __launch_bounds__(MO_THREADS) moe_decode_down_kernel(MoeDecodeArgs a, int slots) {
  pdl_prologue();
  const int b = blockIdx.x, lane = threadIdx.x % WARP, warp = threadIdx.x / WARP;
  const int m = blockIdx.y * MO_WARPS + warp;
  if (m >= a.D) return;
  const T *act = static_cast<const T *>(a.act) + (size_t)b * slots * a.ld_act;
  float acc[1] = {0.f};
  for (int s = 0; s < slots; ++s) {
    const bool shared = s == a.top;
    const int F = shared ? a.F_shared : a.F;
    const T *w = shared ? static_cast<const T *>(a.shared_down) + (size_t)m * F
                        : static_cast<const T *>(a.w_down) + ((size_t)a.chosen[b * a.top + s] * a.D + m) * F;
    warp_rows<T, VEC, 1, 4>(w, 0, act + (size_t)s * a.ld_act, F, acc);
  }
  const float s = warp_sum(acc[0]);
  if (lane == 0) a.y[(size_t)b * a.D + m] = s + (a.init ? a.init[(size_t)b * a.D + m] : 0.f);
}

template <typename T>
static int launch_decode(const MoeDecodeArgs &a, bool up, bool down, cudaStream_t st) {
  const int slots = a.top + (a.shared_gu ? 1 : 0), fmax = a.F > a.F_shared || !a.shared_gu ? a.F : a.F_shared;
  constexpr int N = Chunk<T>::N;
  const bool vec_up = a.D % N == 0 && aligned16(a.x) && aligned16(a.w_gu) && aligned16(a.shared_gu);
  const bool vec_down = a.F % N == 0 && (!a.shared_gu || a.F_shared % N == 0) && a.ld_act % N == 0 && aligned16(a.act) &&
                        aligned16(a.w_down) && aligned16(a.shared_down);
  if (up) {
    const dim3 grid(a.B, ceil_div(fmax, MO_WARPS), slots);
    if (vec_up) djv::launch_kernel(moe_decode_up_kernel<T, true>, grid, dim3(MO_THREADS), 0, st, a);
    else djv::launch_kernel(moe_decode_up_kernel<T, false>, grid, dim3(MO_THREADS), 0, st, a);
    count_launch();
  }
  if (down) {
    const dim3 grid(a.B, ceil_div(a.D, MO_WARPS));
    if (vec_down) djv::launch_kernel(moe_decode_down_kernel<T, true>, grid, dim3(MO_THREADS), 0, st, a, slots);
    else djv::launch_kernel(moe_decode_down_kernel<T, false>, grid, dim3(MO_THREADS), 0, st, a, slots);
    count_launch();
  }
  return check_launch("moe_decode");
}

}  // namespace djv

using namespace djv;

extern "C" int djv_moe_route(int dtype, void *xs, const void *x, const float *z, int *expert, int *place, float *weight,
                             float *ws, int *count, int *offsets, int n, int E, int top, int D, void *stream) {
  DJV_REQUIRE(dtype == DJV_DTYPE_BF16 || dtype == DJV_DTYPE_F32, "moe_route: dtype %d", dtype);
  DJV_REQUIRE(xs && x && z && expert && place && weight && ws && count && offsets, "moe_route: null pointer");
  DJV_REQUIRE(n >= 1 && E >= 1 && E <= MAX_EXPERTS && top >= 1 && top <= E && top <= MAX_TOP && D >= 1 &&
                  (long long)n * top < (1ll << 31),
              "moe_route: n=%d, %d of %d experts, D=%d", n, top, E, D);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (cudaMemsetAsync(count, 0, (size_t)E * 4, st) != cudaSuccess) return check_launch("moe_route");
  djv::launch_kernel(moe_route_kernel, dim3(ceil_div(n, RT_TOKENS)), dim3(RT_WARPS * WARP),
                     4 * (size_t)(2 * E + 2 * RT_TOKENS * top), st, z, n, E, top, expert, place, weight, count);
  const size_t sm = 4 * (size_t)(E + 1);
  const int rows = n * top, most = 8 * sm_count(), grid = rows < most ? rows : most;
  const bool vec = D % (16 / (int)dtype_bytes(dtype)) == 0 && aligned16(x) && aligned16(xs);
#define DJV_GO(T_, V_)                                                                                                \
  djv::launch_kernel(moe_scatter_kernel<T_, V_>, dim3(grid), dim3(256), sm, st, static_cast<T_ *>(xs),                \
                     static_cast<const T_ *>(x), static_cast<const int *>(expert), place,                             \
                     static_cast<const float *>(weight), ws, static_cast<const int *>(count), offsets, n, E, top, D)
  if (dtype == DJV_DTYPE_BF16) {
    if (vec) DJV_GO(bf16, true);
    else DJV_GO(bf16, false);
  } else {
    if (vec) DJV_GO(float, true);
    else DJV_GO(float, false);
  }
#undef DJV_GO
  count_launch(2);
  return check_launch("moe_route");
}

extern "C" int djv_moe_grouped(int dtype, void *y, const void *x, const void *w, const float *scale, const int *offsets,
                               int R, int E, int N, int K, int glu, void *stream) {
  DJV_REQUIRE(dtype == DJV_DTYPE_BF16 || dtype == DJV_DTYPE_F32, "moe_grouped: dtype %d", dtype);
  DJV_REQUIRE(y && x && w && offsets, "moe_grouped: null pointer");
  DJV_REQUIRE(R >= 1 && E >= 1 && E <= MAX_EXPERTS && N >= 1 && K >= 1 && (!glu || N % 2 == 0),
              "moe_grouped: R=%d E=%d N=%d K=%d", R, E, N, K);
  const GroupedArgs a{y, x, w, scale, offsets, R, E, N, K, glu};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (moe_grouped_tc_supported(dtype, a)) return moe_grouped_tc(a, st);
  const long long tiles = (long long)R / GG_M + E;  // no fewer than there can be
  DJV_REQUIRE(tiles <= 65535, "moe_grouped: %d rows are too many", R);
  const dim3 grid(ceil_div(N, GG_N), (unsigned)tiles);
  if (dtype == DJV_DTYPE_BF16) djv::launch_kernel(moe_grouped_kernel<bf16>, grid, dim3(GG_THREADS), 0, st, a);
  else djv::launch_kernel(moe_grouped_kernel<float>, grid, dim3(GG_THREADS), 0, st, a);
  count_launch();
  return check_launch("moe_grouped");
}

extern "C" int djv_moe_decode(int dtype, float *y, void *act, int *chosen, const void *x, const float *z, const void *w_gu,
                              const void *w_down, const void *shared_gu, const void *shared_down, const float *init, int B,
                              int E, int top, int D, int F, int F_shared, int ld_act, int stages, void *stream) {
  DJV_REQUIRE(dtype == DJV_DTYPE_BF16 || dtype == DJV_DTYPE_F32, "moe_decode: dtype %d", dtype);
  DJV_REQUIRE(y && act && chosen && x && z && w_gu && w_down && (!shared_gu) == (!shared_down), "moe_decode: null pointer");
  DJV_REQUIRE(B >= 1 && E >= 1 && top >= 1 && top <= E && top <= MAX_TOP && D >= 1 && F >= 1 && ld_act >= F &&
                  (!shared_gu || (F_shared >= 1 && ld_act >= F_shared)),
              "moe_decode: B=%d, %d of %d experts, D=%d F=%d + %d", B, top, E, D, F, F_shared);
  const MoeDecodeArgs a{y, act, chosen, x, z, w_gu, w_down, shared_gu, shared_down, init, B, E, top, D, F,
                        shared_gu ? F_shared : 0, ld_act};
  DJV_REQUIRE(ceil_div(F > a.F_shared ? F : a.F_shared, MO_WARPS) <= 65535 && ceil_div(D, MO_WARPS) <= 65535,
              "moe_decode: D=%d or F=%d is too large", D, F);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == DJV_DTYPE_BF16 ? launch_decode<bf16>(a, stages & 1, stages & 2, st)
                                 : launch_decode<float>(a, stages & 1, stages & 2, st);
}
