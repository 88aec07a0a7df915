// Routed feed-forward: every token goes through the `top` experts with the largest router scores sigmoid(z); an expert is a
// gated unit whose input is the token's activation times its score.
//
// A prompt portion is sorted by expert on the device (no host synchronisation) and runs as grouped matrix products: this
// file has the sorting and a CUDA-core form of the product for any size, hybrid_moe_gemm.cu the tensor-core form. A decode
// step runs two kernels on the chosen experts' weights; a shared expert, which every token uses, runs in the same two.
#include <cooperative_groups.h>

#include "../../include/dejavu_b200_routed.h"
#include "hybrid_moe.cuh"
#include "mma.cuh"

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
constexpr int RT_WARPS = 8, RT_TOKENS = 16;

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
  const int step = gridDim.x * (blockDim.x / WARP);
  for (int i = blockIdx.x * (blockDim.x / WARP) + tid / WARP; i < n * top; i += step) {  // a warp per row
    const int to = off[expert[i]] + place[i];
    __syncwarp();  // everybody has read place[i]
    if (lane == 0) {
      place[i] = to;
      ws[to] = weight[i];
    }
    const T *src = x + (size_t)(i / top) * D;
    T *dst = xs + (size_t)to * D;
    if (VEC) {
      constexpr int U = 8;
      const int nch = D / Chunk<T>::N;
      for (int c0 = lane; c0 < nch; c0 += WARP * U) {
        uint4 v[U];
#pragma unroll
        for (int u = 0; u < U; ++u)
          if (c0 + u * WARP < nch) v[u] = reinterpret_cast<const uint4 *>(src)[c0 + u * WARP];
#pragma unroll
        for (int u = 0; u < U; ++u)
          if (c0 + u * WARP < nch) reinterpret_cast<uint4 *>(dst)[c0 + u * WARP] = v[u];
      }
    } else {
      for (int c = lane; c < D; c += WARP) dst[c] = src[c];
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

// dot products of R rows of w (stride ld) with x, N elements, by `lanes` lanes of which this is one: U 16-byte chunks per
// lane and row in flight
template <typename T, bool VEC, int R, int U>
__device__ __forceinline__ void warp_rows(const T *w, size_t ld, const T *x, int n, float (&acc)[R], int lane, int lanes) {
  if (VEC) {
    const int nch = n / Chunk<T>::N;
    for (int c0 = lane; c0 < nch; c0 += lanes * U) {
      uint4 v[R][U];
#pragma unroll
      for (int u = 0; u < U; ++u)
#pragma unroll
        for (int r = 0; r < R; ++r) {
          const int c = c0 + u * lanes;
          v[r][u] = c < nch ? ld_stream16(reinterpret_cast<const uint4 *>(w + r * ld) + c) : make_uint4(0, 0, 0, 0);
        }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = c0 + u * lanes;
        if (c < nch) {
          const uint4 xv = *(reinterpret_cast<const uint4 *>(x) + c);
#pragma unroll
          for (int r = 0; r < R; ++r) acc[r] = dot_chunk<T>(v[r][u], xv, acc[r]);
        }
      }
    }
  } else {
    for (int c = lane; c < n; c += lanes)
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
  warp_rows<T, VEC, 2, 4>(w + (size_t)2 * o * a.D, a.D, static_cast<const T *>(a.x) + (size_t)b * a.D, a.D, acc, lane, WARP);
  acc[0] = warp_sum(acc[0]);
  acc[1] = warp_sum(acc[1]);
  if (lane == 0)
    static_cast<T *>(a.act)[((size_t)b * gridDim.z + slot) * a.ld_act + o] = from_f<T>(silu_glu(wt * acc[0], wt * acc[1]));
}

// WPR warps share a row of the result
template <typename T, bool VEC, int WPR>
__global__ void __launch_bounds__(MO_THREADS) moe_decode_down_kernel(MoeDecodeArgs a, int slots) {
  __shared__ float red[MO_WARPS];
  pdl_prologue();
  const int b = blockIdx.x, lane = threadIdx.x % WARP, warp = threadIdx.x / WARP;
  const int m = blockIdx.y * (MO_WARPS / WPR) + warp / WPR, part = warp % WPR;
  const T *act = static_cast<const T *>(a.act) + (size_t)b * slots * a.ld_act;
  float acc[1] = {0.f};
  if (m < a.D)
    for (int s = 0; s < slots; ++s) {
      const bool shared = s == a.top;
      const int F = shared ? a.F_shared : a.F;
      const T *w = shared ? static_cast<const T *>(a.shared_down) + (size_t)m * F
                          : static_cast<const T *>(a.w_down) + ((size_t)a.chosen[b * a.top + s] * a.D + m) * F;
      warp_rows<T, VEC, 1, 4>(w, 0, act + (size_t)s * a.ld_act, F, acc, part * WARP + lane, WPR * WARP);
    }
  float sum = warp_sum(acc[0]);
  if (WPR > 1) {
    if (lane == 0) red[warp] = sum;
    __syncthreads();
    sum = 0.f;
#pragma unroll
    for (int x = 0; x < WPR; ++x) sum += red[warp / WPR * WPR + x];
  }
  if (lane == 0 && part == 0 && m < a.D) a.y[(size_t)b * a.D + m] = sum + (a.init ? a.init[(size_t)b * a.D + m] : 0.f);
}

// ---- decode, several rows: every weight row is read once -----------------------------------------------------------
// mma.sync tiles of 16 weight rows x 8 * NT sequences, the reduction split over the block's warps; weights and activations
// are permuted along it the same way (see rowdot_mma.cuh). A sequence that did not choose the expert takes no part: its
// products are not stored (up), or its activations are zeros (down, which adds up all experts in one accumulator).
constexpr int MM_ROWS_TILE = 16, MM_B = 32;

template <int NT>
__device__ __forceinline__ void mma_chunk(float (&acc)[NT][4], const uint4 &lo, const uint4 &hi, const uint4 (&x)[NT]) {
#pragma unroll
  for (int j = 0; j < NT; ++j) {
    mma_m16n8k16_t<bf16>(acc[j], lo.x, hi.x, lo.y, hi.y, x[j].x, x[j].y);
    mma_m16n8k16_t<bf16>(acc[j], lo.z, hi.z, lo.w, hi.w, x[j].z, x[j].w);
  }
}

template <int NT>  // grid (tiles of 16 gate and up rows, experts and the shared one)
__global__ void __launch_bounds__(MO_THREADS) moe_up_mma_kernel(MoeDecodeArgs a) {
  __shared__ float red[MO_WARPS][NT][MM_ROWS_TILE][8], weight[MM_B];
  __shared__ int slot[MM_B];
  pdl_prologue();
  const int tid = threadIdx.x, warp = tid / WARP, lane = tid % WARP, e = blockIdx.y;
  const bool shared = e == a.E;
  const int rows = 2 * (shared ? a.F_shared : a.F), m0 = blockIdx.x * MM_ROWS_TILE;
  if (m0 >= rows) return;
  bool mine = false;
  for (int b = warp; b < a.B; b += MO_WARPS) {  // the expert's place among the sequence's choices
    int ahead = shared ? a.top : 0;
    float z = 0.f;
    if (!shared) {
      z = a.z[(size_t)b * a.E + e];
      for (int o = lane; o < a.E; o += WARP) {
        const float v = a.z[(size_t)b * a.E + o];
        ahead += v > z || (v == z && o < e);
      }
      ahead = (int)__reduce_add_sync(0xffffffffu, (unsigned)ahead);
    }
    const bool in = shared || ahead < a.top;
    mine |= in;
    if (lane == 0) {
      slot[b] = in ? ahead : -1;
      weight[b] = shared ? 1.f : sigmoid_f(z);
    }
  }
  if (!__syncthreads_or(mine)) return;
  const int g = lane / 4, t = lane % 4;
  const bf16 *W = shared ? static_cast<const bf16 *>(a.shared_gu) : static_cast<const bf16 *>(a.w_gu) + (size_t)e * 2 * a.F * a.D;
  const bool ok_lo = m0 + g < rows, ok_hi = m0 + g + 8 < rows;
  const bf16 *w_lo = W + (size_t)(m0 + g) * a.D, *w_hi = w_lo + (size_t)8 * a.D, *X = static_cast<const bf16 *>(a.x);
  float acc[NT][4] = {};
  constexpr int U = 2;
  const int kblocks = (a.D + 31) / 32;
  for (int kb = warp; kb < kblocks; kb += MO_WARPS * U) {
    uint4 lo[U], hi[U], x[U][NT];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int k = (kb + u * MO_WARPS) * 32 + t * 8;
      const bool ok = k < a.D;
      lo[u] = ok && ok_lo ? ld_stream16(w_lo + k) : make_uint4(0, 0, 0, 0);
      hi[u] = ok && ok_hi ? ld_stream16(w_hi + k) : make_uint4(0, 0, 0, 0);
#pragma unroll
      for (int j = 0; j < NT; ++j)
        x[u][j] = ok && j * 8 + g < a.B ? ld_cached16(X + (size_t)(j * 8 + g) * a.D + k) : make_uint4(0, 0, 0, 0);
    }
#pragma unroll
    for (int u = 0; u < U; ++u) mma_chunk<NT>(acc, lo[u], hi[u], x[u]);
  }
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int x = 0; x < 4; ++x) red[warp][j][g + (x / 2) * 8][2 * t + x % 2] = acc[j][x];
  __syncthreads();
  const int slots = a.top + (a.shared_gu ? 1 : 0);
  for (int o = tid; o < NT * MM_ROWS_TILE / 2 * 8; o += MO_THREADS) {  // (sequence group, gated unit, sequence)
    const int c = o % 8, r = o / 8 % (MM_ROWS_TILE / 2) * 2, j = o / (MM_ROWS_TILE / 2 * 8), b = j * 8 + c;
    if (b >= a.B || slot[b] < 0 || m0 + r >= rows) continue;
    float gate = 0.f, up = 0.f;
#pragma unroll
    for (int w = 0; w < MO_WARPS; ++w) {
      gate += red[w][j][r][c];
      up += red[w][j][r + 1][c];
    }
    static_cast<bf16 *>(a.act)[((size_t)b * slots + slot[b]) * a.ld_act + (m0 + r) / 2] =
        from_f<bf16>(silu_glu(weight[b] * gate, weight[b] * up));
  }
}

template <int NT>  // grid (tiles of 16 rows, S), a cluster over the S parts of the reduction
__global__ void __launch_bounds__(MO_THREADS) moe_down_mma_kernel(MoeDecodeArgs a, int slots) {
  extern __shared__ int sm[];
  __shared__ float red[MO_WARPS][NT][MM_ROWS_TILE][8], part[NT][MM_ROWS_TILE][8];
  __shared__ int n_list;
  pdl_prologue();
  const int tid = threadIdx.x, warp = tid / WARP, lane = tid % WARP, S = gridDim.y, sb = blockIdx.y;
  int *list = sm;                                            // [E]: experts that any sequence chose
  signed char *place = reinterpret_cast<signed char *>(list + a.E);  // [E][MM_B]: the expert's place among a sequence's choices
  for (int i = tid; i < a.E * MM_B / 4; i += MO_THREADS) reinterpret_cast<int *>(place)[i] = -1;
  __syncthreads();
  for (int b = warp; b < a.B; b += MO_WARPS) {
    int e;
    float v;
    warp_topk(a.z + (size_t)b * a.E, a.E, a.top, e, v);
    if (lane < a.top) place[e * MM_B + b] = (signed char)lane;
  }
  __syncthreads();
  if (warp == 0) {
    int n = 0;
    for (int e0 = 0; e0 < a.E; e0 += WARP) {
      bool used = false;
      if (e0 + lane < a.E)
        for (int b = 0; b < a.B; ++b) used |= place[(e0 + lane) * MM_B + b] >= 0;
      const unsigned mask = __ballot_sync(0xffffffffu, used);
      if (used) list[n + __popc(mask & ((1u << lane) - 1))] = e0 + lane;
      n += __popc(mask);
    }
    if (lane == 0) n_list = n;
  }
  __syncthreads();
  const int g = lane / 4, t = lane % 4, m0 = blockIdx.x * MM_ROWS_TILE;
  const bool ok_lo = m0 + g < a.D, ok_hi = m0 + g + 8 < a.D;
  // blocks of 32 reduction elements of all experts in a row, then the shared one's
  const int kf = (a.F + 31) / 32, routed = n_list * kf, total = routed + (slots > a.top ? (a.F_shared + 31) / 32 : 0);
  const bf16 *act = static_cast<const bf16 *>(a.act);
  float acc[NT][4] = {};
  constexpr int U = NT == 1 ? 4 : 2;
  const int stride = MO_WARPS * S;
  for (int i0 = sb * MO_WARPS + warp; i0 < total; i0 += stride * U) {
    uint4 lo[U], hi[U], x[U][NT];
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const int i = i0 + u * stride;
      lo[u] = hi[u] = make_uint4(0, 0, 0, 0);
#pragma unroll
      for (int j = 0; j < NT; ++j) x[u][j] = make_uint4(0, 0, 0, 0);
      if (i >= total) continue;
      const bool shared = i >= routed;
      const int at = shared ? 0 : i / kf, k = (i - (shared ? routed : at * kf)) * 32 + t * 8;
      const int F = shared ? a.F_shared : a.F, e = shared ? 0 : list[at];
      if (k >= F) continue;
      const bf16 *w = (shared ? static_cast<const bf16 *>(a.shared_down) : static_cast<const bf16 *>(a.w_down) + (size_t)e * a.D * F) +
                      (size_t)(m0 + g) * F + k;
      if (ok_lo) lo[u] = ld_stream16(w);
      if (ok_hi) hi[u] = ld_stream16(w + (size_t)8 * F);
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        const int b = j * 8 + g, s = b >= a.B ? -1 : (shared ? a.top : place[e * MM_B + b]);
        if (s >= 0) x[u][j] = *reinterpret_cast<const uint4 *>(act + ((size_t)b * slots + s) * a.ld_act + k);
      }
    }
#pragma unroll
    for (int u = 0; u < U; ++u) mma_chunk<NT>(acc, lo[u], hi[u], x[u]);
  }
#pragma unroll
  for (int j = 0; j < NT; ++j)
#pragma unroll
    for (int x = 0; x < 4; ++x) red[warp][j][g + (x / 2) * 8][2 * t + x % 2] = acc[j][x];
  __syncthreads();
  for (int o = tid; o < NT * MM_ROWS_TILE * 8; o += MO_THREADS) {
    const int c = o % 8, r = o / 8 % MM_ROWS_TILE, j = o / (MM_ROWS_TILE * 8);
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < MO_WARPS; ++w) s += red[w][j][r][c];
    part[j][r][c] = s;
  }
  cooperative_groups::cluster_group cluster = cooperative_groups::this_cluster();
  if (S > 1) cluster.sync();
  else __syncthreads();
  if (sb == 0)
    for (int o = tid; o < NT * MM_ROWS_TILE * 8; o += MO_THREADS) {
      const int r = o % MM_ROWS_TILE, c = o / MM_ROWS_TILE % 8, j = o / (MM_ROWS_TILE * 8), b = j * 8 + c, m = m0 + r;
      if (b >= a.B || m >= a.D) continue;
      float s = a.init ? a.init[(size_t)b * a.D + m] : 0.f;
      for (int q = 0; q < S; ++q) s += S > 1 ? cluster.map_shared_rank(&part[0][0][0], q)[(j * MM_ROWS_TILE + r) * 8 + c] : part[j][r][c];
      a.y[(size_t)b * a.D + m] = s;
    }
  if (S > 1) cluster.sync();  // no block leaves while block 0 may still read its sums
}

template <int NT>
static void launch_mma(const MoeDecodeArgs &a, int slots, int fmax, bool up, bool down, cudaStream_t st) {
  if (up) {
    djv::launch_kernel(moe_up_mma_kernel<NT>, dim3(ceil_div(2 * fmax, MM_ROWS_TILE), a.E + (a.shared_gu ? 1 : 0)), dim3(MO_THREADS),
                       0, st, a);
    count_launch();
  }
  if (down) {
    const int tiles = ceil_div(a.D, MM_ROWS_TILE);
    int S = 1;
    while (S < 8 && tiles * S < 4 * sm_count()) S *= 2;
    djv::launch_kernel_cluster(moe_down_mma_kernel<NT>, dim3(tiles, S), dim3(MO_THREADS), (size_t)a.E * (4 + MM_B), st,
                               dim3(1, S, 1), a, slots);
    count_launch();
  }
}

template <typename T>
static int launch_decode(const MoeDecodeArgs &a, bool up, bool down, cudaStream_t st) {
  const int slots = a.top + (a.shared_gu ? 1 : 0), fmax = a.F > a.F_shared || !a.shared_gu ? a.F : a.F_shared;
  constexpr int N = Chunk<T>::N;
  const bool vec_up = a.D % N == 0 && aligned16(a.x) && aligned16(a.w_gu) && aligned16(a.shared_gu);
  const bool vec_down = a.F % N == 0 && (!a.shared_gu || a.F_shared % N == 0) && a.ld_act % N == 0 && aligned16(a.act) &&
                        aligned16(a.w_down) && aligned16(a.shared_down);
  if constexpr (sizeof(T) == 2) {
    // several rows share weights (both stages take this form or neither: they agree on where a choice's activations are)
    if (a.B >= 2 && a.B <= MM_B && vec_up && vec_down && (size_t)a.E * (4 + MM_B) <= 40 * 1024) {
      switch ((a.B + 7) / 8) {
        case 1: launch_mma<1>(a, slots, fmax, up, down, st); break;
        case 2: launch_mma<2>(a, slots, fmax, up, down, st); break;
        case 3: launch_mma<3>(a, slots, fmax, up, down, st); break;
        default: launch_mma<4>(a, slots, fmax, up, down, st); break;
      }
      return check_launch("moe_decode");
    }
  }
  if (up) {
    const dim3 grid(a.B, ceil_div(fmax, MO_WARPS), slots);
    if (vec_up) djv::launch_kernel(moe_decode_up_kernel<T, true>, grid, dim3(MO_THREADS), 0, st, a);
    else djv::launch_kernel(moe_decode_up_kernel<T, false>, grid, dim3(MO_THREADS), 0, st, a);
    count_launch();
  }
  if (down) {
    // as many warps per row as still lets every block be resident at once and gives each lane work
    int wpr = 1;
    while (wpr < 4 && (long long)a.B * a.D * wpr * 2 <= (long long)8 * MO_WARPS * sm_count() && a.F / N >= WARP * wpr * 2) wpr *= 2;
    const dim3 grid(a.B, ceil_div(a.D, MO_WARPS / wpr));
    if (!vec_down) djv::launch_kernel(moe_decode_down_kernel<T, false, 1>, dim3(a.B, ceil_div(a.D, MO_WARPS)), dim3(MO_THREADS), 0, st, a, slots);
    else if (wpr == 1) djv::launch_kernel(moe_decode_down_kernel<T, true, 1>, grid, dim3(MO_THREADS), 0, st, a, slots);
    else if (wpr == 2) djv::launch_kernel(moe_decode_down_kernel<T, true, 2>, grid, dim3(MO_THREADS), 0, st, a, slots);
    else djv::launch_kernel(moe_decode_down_kernel<T, true, 4>, grid, dim3(MO_THREADS), 0, st, a, slots);
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
  const int blocks = ceil_div(n * top, 8), most = 8 * sm_count(), grid = blocks < most ? blocks : most;
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
