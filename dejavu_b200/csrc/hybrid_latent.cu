// Latent attention: keys and values of all heads are projections of one latent per token, and a rotated key part is
// shared by the heads, so the cache holds (latent, rotated part) rows and nothing else:
//   ring (B, cap, rank + rot): position p of a sequence sits in slot p % cap.
//
// A portion of tokens expands the latents it can see into keys and values with one matrix product and runs the windowed
// attention kernels on them. A decode step leaves the latents as they are: the key projection is applied to the query
// and the value projection to the weighted sum of latents, so that every head reads the same rows.
#include <math.h>

#include "../../include/dejavu_b200_routed.h"
#include "hybrid_attention.cuh"
#include "hybrid_latent.cuh"

namespace djv {

// blocks among which the sequences of a decode step are dealt out, per block of weights
constexpr int LATENT_GROUPS = 8;

// one row: RMS norm of the latent, rotation of the shared key part, by a whole block
template <typename T>
__device__ __forceinline__ void make_latent_row(const T *src, T *dst, const float *norm, float eps, const float *freqs,
                                                long long pos, int rank, int rot) {
  __shared__ float red[32];
  const int tid = threadIdx.x, warps = blockDim.x / WARP;
  float ss = 0.f;
  for (int i = tid; i < rank; i += blockDim.x) {
    const float v = to_f(src[i]);
    ss = fmaf(v, v, ss);
  }
  ss = warp_sum(ss);
  if (tid % WARP == 0) red[tid / WARP] = ss;
  __syncthreads();
  float tot = 0.f;
  for (int w = 0; w < warps; ++w) tot += red[w];
  const float r = 1.f / sqrtf(tot / (float)rank + eps);
  for (int i = tid; i < rank; i += blockDim.x) dst[i] = from_f<T>(to_f(src[i]) * r * norm[i]);
  for (int i = tid; i < rot / 2; i += blockDim.x) {
    float s, c;
    sincosf((float)pos * freqs[i], &s, &c);
    const float u = to_f(src[rank + 2 * i]), v = to_f(src[rank + 2 * i + 1]);
    dst[rank + 2 * i] = from_f<T>(u * c - v * s);
    dst[rank + 2 * i + 1] = from_f<T>(v * c + u * s);
  }
  __syncthreads();  // red[] may be used again
}

// ---- prompt portions: rows of the earlier tokens that are in sight, then the portion's own -------------------------
template <typename T>
__global__ void latent_rows_kernel(T *__restrict__ rows, const T *__restrict__ src, long long ld,
                                   const T *__restrict__ ring, const float *__restrict__ norm, float eps,
                                   const float *__restrict__ freqs, const long long *__restrict__ pos, int n, int past,
                                   int rank, int rot, int cap) {
  pdl_prologue();
  const int j = (int)blockIdx.x - past, b = blockIdx.y, w = rank + rot;
  T *dst = rows + ((size_t)b * (past + n) + blockIdx.x) * w;
  const long long p = pos[b] + j;
  if (j >= 0) {
    make_latent_row<T>(src + ((size_t)b * n + j) * ld, dst, norm, eps, freqs, p, rank, rot);
    return;
  }
  const T *old = p >= 0 ? ring + ((size_t)b * cap + (size_t)(p % cap)) * w : nullptr;
  for (int i = threadIdx.x; i < w; i += blockDim.x) dst[i] = old ? old[i] : from_f<T>(0.f);
}

// the same with 16-byte accesses, a warp per row of at most LR_U * 32 latent chunks; with `store` (only where no earlier
// rows are read) the new rows also enter the ring
constexpr int LR_WARPS = 4, LR_U = 4;
template <typename T>
__global__ void __launch_bounds__(LR_WARPS * WARP)
latent_rows_warp_kernel(T *__restrict__ rows, const T *__restrict__ src, long long ld, T *__restrict__ ring,
                        const float *__restrict__ norm, float eps, const float *__restrict__ freqs,
                        const long long *__restrict__ pos, int n, int past, int rank, int rot, int cap, int store) {
  pdl_prologue();
  constexpr int N = Chunk<T>::N;
  const int lane = threadIdx.x % WARP, row = blockIdx.x * LR_WARPS + threadIdx.x / WARP, b = blockIdx.y;
  if (row >= past + n) return;
  const int j = row - past, w = rank + rot, nch = rank / N;
  T *dst = rows + ((size_t)b * (past + n) + row) * w;
  const long long p = pos[b] + j;
  if (j < 0) {
    const uint4 *old = p >= 0 ? reinterpret_cast<const uint4 *>(ring + ((size_t)b * cap + (size_t)(p % cap)) * w) : nullptr;
    for (int c = lane; c < w / N; c += WARP) reinterpret_cast<uint4 *>(dst)[c] = old ? old[c] : make_uint4(0, 0, 0, 0);
    return;
  }
  T *slot = store && j >= n - cap ? ring + ((size_t)b * cap + (size_t)(p % cap)) * w : nullptr;
  const T *s = src + ((size_t)b * n + j) * ld;
  float f[LR_U][N], ss = 0.f;
#pragma unroll
  for (int u = 0; u < LR_U; ++u) {
    const int c = lane + u * WARP;
    const uint4 v = c < nch ? reinterpret_cast<const uint4 *>(s)[c] : make_uint4(0, 0, 0, 0);
    unpack_chunk<T>(v, f[u]);
  }
#pragma unroll
  for (int u = 0; u < LR_U; ++u)
#pragma unroll
    for (int e = 0; e < N; ++e) ss = fmaf(f[u][e], f[u][e], ss);
  const float r = 1.f / sqrtf(warp_sum(ss) / (float)rank + eps);
#pragma unroll
  for (int u = 0; u < LR_U; ++u) {
    const int c = lane + u * WARP;
    if (c >= nch) continue;
    T o[N];
#pragma unroll
    for (int e = 0; e < N; ++e) o[e] = from_f<T>(f[u][e] * r * norm[c * N + e]);
    reinterpret_cast<uint4 *>(dst)[c] = *reinterpret_cast<uint4 *>(o);
    if (slot) reinterpret_cast<uint4 *>(slot)[c] = *reinterpret_cast<uint4 *>(o);
  }
  for (int i = lane; i < rot / 2; i += WARP) {
    float sn, cs;
    sincosf((float)p * freqs[i], &sn, &cs);
    const float u = to_f(s[rank + 2 * i]), v = to_f(s[rank + 2 * i + 1]);
    const T x = from_f<T>(u * cs - v * sn), y = from_f<T>(v * cs + u * sn);
    dst[rank + 2 * i] = x;
    dst[rank + 2 * i + 1] = y;
    if (slot) {
      slot[rank + 2 * i] = x;
      slot[rank + 2 * i + 1] = y;
    }
  }
}

// the new rows enter the ring (after latent_rows_kernel has read the old ones): the last min(n, cap) tokens
template <typename T>
__global__ void latent_store_kernel(T *__restrict__ ring, const T *__restrict__ rows, const long long *__restrict__ pos,
                                    int n, int past, int width, int cap, int first) {
  pdl_prologue();
  const int t = first + blockIdx.x, b = blockIdx.y;
  const T *src = rows + ((size_t)b * (past + n) + past + t) * width;
  T *dst = ring + ((size_t)b * cap + (size_t)((pos[b] + t) % cap)) * width;
  for (int i = threadIdx.x; i < width; i += blockDim.x) dst[i] = src[i];
}

// ---- decode: queries ------------------------------------------------------------------------------------------------
// Blocks 0 .. H * cbs - 1: query of head h against columns of its key projection, for all sequences,
//   out[b, h, r] = sum_d q[b, h, d] uk[h * dim + d, r];  the first column block of a head also rotates its query part.
// The blocks after them: a sequence's new latent row goes straight into its ring slot.
// V columns per thread; with REG the weights (at most LQ_REG rows per thread) are fetched before the kernel waits for its
// predecessor and stay in registers for the block's `per` sequences.
template <typename T, int V, bool REG>
__global__ void __launch_bounds__(LQ_THREADS) latent_query_kernel(LatentDecodeArgs a, int cbs, int per) {
  extern __shared__ float sm[];
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  constexpr int CT = LQ_COLS / V, RG = LQ_THREADS / CT;  // threads along the columns, row groups
  const int tid = threadIdx.x, w = a.rank + a.rot, qd = a.dim + a.rot;
  const int b0 = blockIdx.y * per, b1 = min(a.B, b0 + per);
  if ((int)blockIdx.x >= a.H * cbs) {
    asm volatile("griddepcontrol.wait;" ::: "memory");
    const int b = b0 + blockIdx.x - a.H * cbs;
    if (b >= b1) return;
    const long long p = a.pos[b];
    make_latent_row<T>(static_cast<const T *>(a.proj) + (size_t)b * a.ld + (size_t)a.H * qd,
                       static_cast<T *>(a.ring) + ((size_t)b * a.cap + (size_t)(p % a.cap)) * w, a.norm, a.eps, a.freqs, p,
                       a.rank, a.rot);
    return;
  }
  const int h = blockIdx.x / cbs, c0 = (blockIdx.x % cbs) * LQ_COLS;
  const int col = c0 + tid % CT * V, rg = tid / CT;
  const bool mine = col < a.rank;
  const T *W = static_cast<const T *>(a.uk) + (size_t)h * a.dim * a.rank + col;
  uint4 wr[REG ? LQ_REG : 1];
  if constexpr (REG) {
#pragma unroll
    for (int x = 0; x < LQ_REG; ++x) {
      const int d = rg + x * RG;
      wr[x] = mine && d < a.dim ? ld_stream16(W + (size_t)d * a.rank) : make_uint4(0, 0, 0, 0);
    }
  }
  asm volatile("griddepcontrol.wait;" ::: "memory");
  float *q = sm, *red = q + ((a.dim + 3) & ~3);  // [RG][LQ_COLS]
  for (int b = b0; b < b1; ++b) {
    const T *row = static_cast<const T *>(a.proj) + (size_t)b * a.ld + (size_t)h * qd;
    T *out = static_cast<T *>(a.qc) + ((size_t)b * a.H + h) * w;
    for (int i = tid; i < a.dim; i += LQ_THREADS) q[i] = to_f(row[i]);
    __syncthreads();
    float acc[V];
#pragma unroll
    for (int e = 0; e < V; ++e) acc[e] = 0.f;
    if constexpr (REG) {
#pragma unroll
      for (int x = 0; x < LQ_REG; ++x) {
        const int d = rg + x * RG;
        float f[V];
        unpack_chunk<T>(wr[x], f);
        const float qv = d < a.dim ? q[d] : 0.f;
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = fmaf(qv, f[e], acc[e]);
      }
    } else if (mine) {
      for (int d = rg; d < a.dim; d += RG)
#pragma unroll
        for (int e = 0; e < V; ++e) acc[e] = fmaf(q[d], to_f(W[(size_t)d * a.rank + e]), acc[e]);
    }
#pragma unroll
    for (int e = 0; e < V; ++e) red[rg * LQ_COLS + tid % CT * V + e] = acc[e];
    __syncthreads();
    for (int c = tid; c < LQ_COLS; c += LQ_THREADS) {
      if (c0 + c >= a.rank) continue;
      float s = 0.f;
#pragma unroll
      for (int x = 0; x < RG; ++x) s += red[x * LQ_COLS + c];
      out[c0 + c] = from_f<T>(s);
    }
    if (c0 == 0) {
      const float p = (float)a.pos[b];
      for (int i = tid; i < a.rot / 2; i += LQ_THREADS) {
        float s, c;
        sincosf(p * a.freqs[i], &s, &c);
        const float u = to_f(row[a.dim + 2 * i]), v = to_f(row[a.dim + 2 * i + 1]);
        out[a.rank + 2 * i] = from_f<T>(u * c - v * s);
        out[a.rank + 2 * i + 1] = from_f<T>(v * c + u * s);
      }
    }
    __syncthreads();  // q[] and red[] are reused
  }
}

// ---- decode: attention over the latents, any element type and size ------------------------------------------------
// a block per (head, sequence): scores a warp per token, sums a thread per column
constexpr int LS_THREADS = 256, LS_TILE = 128;
template <typename T>
__global__ void __launch_bounds__(LS_THREADS) latent_attend_simple_kernel(LatentDecodeArgs a) {
  extern __shared__ float sm[];
  __shared__ float sc[LS_TILE], m_run, l_run, corr;
  pdl_prologue();
  const int tid = threadIdx.x, lane = tid % WARP, warp = tid / WARP;
  const int h = blockIdx.x, b = blockIdx.y, w = a.rank + a.rot;
  float *q = sm, *o = q + w;
  const T *qr = static_cast<const T *>(a.qc) + ((size_t)b * a.H + h) * w;
  for (int i = tid; i < w; i += LS_THREADS) q[i] = to_f(qr[i]);
  for (int i = tid; i < a.rank; i += LS_THREADS) o[i] = 0.f;
  if (tid == 0) {
    m_run = -INFINITY;
    l_run = 0.f;
  }
  const long long p = a.pos[b];
  long long lo = p - a.window + 1;
  if (lo < 0) lo = 0;
  const T *ring = static_cast<const T *>(a.ring) + (size_t)b * a.cap * w;
  __syncthreads();
  for (long long j0 = lo; j0 <= p; j0 += LS_TILE) {
    const int cnt = (int)min((long long)LS_TILE, p - j0 + 1);
    for (int t = warp; t < cnt; t += LS_THREADS / WARP) {
      const T *k = ring + (size_t)((j0 + t) % a.cap) * w;
      float s = 0.f;
      for (int i = lane; i < w; i += WARP) s = fmaf(q[i], to_f(k[i]), s);
      s = warp_sum(s);
      if (lane == 0) sc[t] = s * a.scale;
    }
    __syncthreads();
    if (warp == 0) {
      float mx = m_run;
      for (int t = lane; t < cnt; t += WARP) mx = fmaxf(mx, sc[t]);
      mx = warp_max(mx);
      float sum = 0.f;
      for (int t = lane; t < cnt; t += WARP) {
        const float e = expf(sc[t] - mx);
        sc[t] = e;
        sum += e;
      }
      sum = warp_sum(sum);
      if (lane == 0) {
        corr = m_run == -INFINITY ? 0.f : expf(m_run - mx);
        l_run = l_run * corr + sum;
        m_run = mx;
      }
    }
    __syncthreads();
    for (int i = tid; i < a.rank; i += LS_THREADS) {
      float v = o[i] * corr;
      for (int t = 0; t < cnt; ++t) v = fmaf(sc[t], to_f(ring[(size_t)((j0 + t) % a.cap) * w + i]), v);
      o[i] = v;
    }
    __syncthreads();
  }
  float *out = a.part_o + ((size_t)b * a.H + h) * a.splits * a.rank, *ml = a.part_ml + ((size_t)b * a.H + h) * a.splits * 2;
  for (int i = tid; i < a.rank; i += LS_THREADS) out[i] = o[i];
  for (int s = tid; s < a.splits; s += LS_THREADS) {  // one part has it all
    ml[2 * s] = s ? -INFINITY : m_run;
    ml[2 * s + 1] = s ? 0.f : l_run;
  }
}

// ---- decode: values -------------------------------------------------------------------------------------------------
// out[b, h, j] = (uv[h * dv + j, :] . ctx[b, h, :]) * sigmoid(gate[b, h, j]), ctx the window's parts put together. A block
// takes LO_ROWS rows per warp of one head and `per` sequences; the weights are fetched before the kernel waits (U 16-byte chunks per lane and
// row).
constexpr int LO_THREADS = 256, LO_WARPS = LO_THREADS / WARP, LO_ROWS = 4;
template <typename T, int U>  // U == 0: any rank and alignment
__global__ void __launch_bounds__(LO_THREADS, U > 2 ? 1 : 2) latent_out_kernel(LatentDecodeArgs a, int per) {
  extern __shared__ __align__(16) float ctx[];  // [2][rank]: two partial sums
  __shared__ float factor[LD_MAX_SPLITS];
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  const int tid = threadIdx.x, lane = tid % WARP, warp = tid / WARP, h = blockIdx.y;
  const int r0 = (blockIdx.x * LO_WARPS + warp) * LO_ROWS, rows = max(0, min(LO_ROWS, a.dv - r0));
  const T *W = static_cast<const T *>(a.uv) + ((size_t)h * a.dv + r0) * a.rank;
  constexpr int N = Chunk<T>::N;
  const int nch = a.rank / N;
  uint4 w[LO_ROWS][U > 0 ? U : 1];
  if constexpr (U > 0) {
#pragma unroll
    for (int r = 0; r < LO_ROWS; ++r)
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = lane + u * WARP;
        w[r][u] = r < rows && c < nch ? ld_stream16(W + (size_t)r * a.rank + c * N) : make_uint4(0, 0, 0, 0);
      }
  }
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const int b1 = min(a.B, ((int)blockIdx.z + 1) * per);
  for (int b = blockIdx.z * per; b < b1; ++b) {
    const size_t bh = (size_t)b * a.H + h;
    if (warp == 0) {  // (at most a part per lane)
      const float m = lane < a.splits ? a.part_ml[(bh * a.splits + lane) * 2] : -INFINITY;
      const float l = lane < a.splits ? a.part_ml[(bh * a.splits + lane) * 2 + 1] : 0.f;
      const float top = warp_max(m), f = m == -INFINITY ? 0.f : expf(m - top);
      factor[lane] = f / warp_sum(f * l);
    }
    __syncthreads();
    const float *part = a.part_o + bh * a.splits * a.rank;
    if (U > 0) {
      // two halves of the block take every other part, 4 columns per thread
      constexpr int HALF = LO_THREADS / 2;
      float *dst = ctx + tid / HALF * a.rank;
      for (int c = tid % HALF * 4; c < a.rank; c += HALF * 4) {
        float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int s = tid / HALF; s < a.splits; s += 2) {
          const float f = factor[s];  // (0: an empty part, whose sums may be anything)
          const float4 v = f != 0.f ? *reinterpret_cast<const float4 *>(part + (size_t)s * a.rank + c) : make_float4(0.f, 0.f, 0.f, 0.f);
          o.x = fmaf(f, v.x, o.x);
          o.y = fmaf(f, v.y, o.y);
          o.z = fmaf(f, v.z, o.z);
          o.w = fmaf(f, v.w, o.w);
        }
        *reinterpret_cast<float4 *>(dst + c) = o;
      }
    } else {
      for (int c = tid; c < a.rank; c += LO_THREADS) {
        float o = 0.f;
        for (int s = 0; s < a.splits; ++s)
          if (factor[s] != 0.f) o = fmaf(factor[s], part[(size_t)s * a.rank + c], o);
        ctx[c] = o;
      }
    }
    __syncthreads();
    float acc[LO_ROWS];
#pragma unroll
    for (int r = 0; r < LO_ROWS; ++r) acc[r] = 0.f;
    if constexpr (U > 0) {
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int c = lane + u * WARP;
        if (c < nch) {
          float xv[N];
#pragma unroll
          for (int e = 0; e < N; e += 4) {
            const float4 u0 = *reinterpret_cast<const float4 *>(ctx + c * N + e);
            const float4 u1 = *reinterpret_cast<const float4 *>(ctx + a.rank + c * N + e);
            xv[e] = u0.x + u1.x;
            xv[e + 1] = u0.y + u1.y;
            xv[e + 2] = u0.z + u1.z;
            xv[e + 3] = u0.w + u1.w;
          }
#pragma unroll
          for (int r = 0; r < LO_ROWS; ++r) {
            float f[N];
            unpack_chunk<T>(w[r][u], f);
#pragma unroll
            for (int e = 0; e < N; ++e) acc[r] = fmaf(f[e], xv[e], acc[r]);
          }
        }
      }
    } else {
      for (int c = lane; c < a.rank; c += WARP)
        for (int r = 0; r < rows; ++r) acc[r] = fmaf(to_f(W[(size_t)r * a.rank + c]), ctx[c], acc[r]);
    }
#pragma unroll
    for (int r = 0; r < LO_ROWS; ++r) acc[r] = warp_sum(acc[r]);
    if (lane < rows) {
      float v = acc[0];
#pragma unroll
      for (int r = 1; r < LO_ROWS; ++r)
        if (lane == r) v = acc[r];
      const size_t col = (size_t)h * a.dv + r0 + lane;
      if (a.gate) v *= sigmoid_f(to_f(static_cast<const T *>(a.gate)[(size_t)b * a.ldg + col]));
      static_cast<T *>(a.out)[(size_t)b * a.H * a.dv + col] = from_f<T>(v);
    }
    if (b + 1 < b1) __syncthreads();  // ctx is reused
  }
}

template <typename T>
static int launch_query(const LatentDecodeArgs &a, cudaStream_t st) {
  constexpr int N = Chunk<T>::N;
  const int cbs = ceil_div(a.rank, LQ_COLS);
  const bool vec = a.rank % N == 0 && aligned16(a.uk);
  const int per = ceil_div(a.B, LATENT_GROUPS);
  const dim3 grid(a.H * cbs + per, ceil_div(a.B, per));
  auto smem = [&](int v) { return 4 * ((size_t)((a.dim + 3) & ~3) + (size_t)(LQ_THREADS / (LQ_COLS / v)) * LQ_COLS); };
  if (vec && a.dim <= LQ_REG * (LQ_THREADS / (LQ_COLS / N)))
    djv::launch_kernel(latent_query_kernel<T, N, true>, grid, dim3(LQ_THREADS), smem(N), st, a, cbs, per);
  else
    djv::launch_kernel(latent_query_kernel<T, 1, false>, grid, dim3(LQ_THREADS), smem(1), st, a, cbs, per);
  count_launch();
  return check_launch("latent_decode");
}

template <typename T>
static int launch_attend(const LatentDecodeArgs &a, cudaStream_t st) {
  if (latent_attend_mma_supported(a, sizeof(T) == 2)) return latent_attend_mma(a, st);
  const size_t smem = 4 * (size_t)(2 * a.rank + a.rot);
  if (smem > 48 * 1024)
    cudaFuncSetAttribute(latent_attend_simple_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  djv::launch_kernel(latent_attend_simple_kernel<T>, dim3(a.H, a.B), dim3(LS_THREADS), smem, st, a);
  count_launch();
  return check_launch("latent_decode");
}

template <typename T>
static int launch_out(const LatentDecodeArgs &a, cudaStream_t st) {
  constexpr int N = Chunk<T>::N;
  const int per = ceil_div(a.B, LATENT_GROUPS);
  const dim3 grid(ceil_div(a.dv, LO_WARPS * LO_ROWS), a.H, ceil_div(a.B, per));
  int u = a.rank % N == 0 && aligned16(a.uv) && aligned16(a.part_o) ? ceil_div(a.rank / N, WARP) : 0;
  if (u > 4) u = 0;
  const size_t smem = (size_t)a.rank * (u ? 8 : 4);
  if (u == 1) djv::launch_kernel(latent_out_kernel<T, 1>, grid, dim3(LO_THREADS), smem, st, a, per);
  else if (u == 2) djv::launch_kernel(latent_out_kernel<T, 2>, grid, dim3(LO_THREADS), smem, st, a, per);
  else if (u == 3 || u == 4) djv::launch_kernel(latent_out_kernel<T, 4>, grid, dim3(LO_THREADS), smem, st, a, per);
  else djv::launch_kernel(latent_out_kernel<T, 0>, grid, dim3(LO_THREADS), smem, st, a, per);
  count_launch();
  return check_launch("latent_decode");
}

}  // namespace djv

using namespace djv;

static int check_latent(const char *op, int dtype, int B, int n, int rank, int rot, int cap) {
  DJV_REQUIRE(dtype == DJV_DTYPE_BF16 || dtype == DJV_DTYPE_F32, "%s: dtype %d", op, dtype);
  DJV_REQUIRE(B >= 1 && B <= 65535 && n >= 1, "%s: B=%d n=%d", op, B, n);
  DJV_REQUIRE(rank >= 1 && rank <= 8192 && rot >= 0 && rot % 2 == 0 && rot <= 8192, "%s: rank %d, %d rotated", op, rank, rot);
  DJV_REQUIRE(cap >= 1, "%s: cap=%d", op, cap);
  return DJV_OK;
}

extern "C" int djv_latent_rows(int dtype, void *rows, const void *proj, long long ld, void *ring, const float *norm,
                               float eps, const float *freqs, const long long *pos, int B, int n, int past, int rank,
                               int rot, int cap, int store, void *stream) {
  int rc = check_latent("latent_rows", dtype, B, n, rank, rot, cap);
  if (rc) return rc;
  DJV_REQUIRE(rows && proj && ring && norm && pos && (freqs || rot == 0), "latent_rows: null pointer");
  DJV_REQUIRE(past >= 0 && past <= cap && ld >= rank + rot, "latent_rows: past=%d cap=%d row stride %lld", past, cap, ld);
  DJV_REQUIRE(store >= 0 && store <= 2 && (store != 2 || past == 0), "latent_rows: store=%d past=%d", store, past);
  const int cnt = n < cap ? n : cap, chunk = 16 / (int)dtype_bytes(dtype);
  const bool vec = rank % chunk == 0 && rot % chunk == 0 && rank / chunk <= LR_U * WARP && ld % chunk == 0 &&
                   aligned16(rows) && aligned16(proj) && aligned16(ring);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
#define DJV_GO(T_)                                                                                                       \
  {                                                                                                                      \
    T_ *r = static_cast<T_ *>(rows), *g = static_cast<T_ *>(ring);                                                       \
    const T_ *p = static_cast<const T_ *>(proj);                                                                         \
    if (store != 1 && vec)                                                                                               \
      djv::launch_kernel(latent_rows_warp_kernel<T_>, dim3(ceil_div(past + n, LR_WARPS), B), dim3(LR_WARPS * WARP), 0,   \
                         st, r, p, ld, g, norm, eps, freqs, pos, n, past, rank, rot, cap, store);                        \
    else if (store != 1)                                                                                                 \
      djv::launch_kernel(latent_rows_kernel<T_>, dim3(past + n, B), dim3(128), 0, st, r, p, ld, g, norm, eps, freqs,     \
                         pos, n, past, rank, rot, cap);                                                                  \
    if (store == 1 || (store == 2 && !vec))                                                                              \
      djv::launch_kernel(latent_store_kernel<T_>, dim3(cnt, B), dim3(128), 0, st, g, r, pos, n, past, rank + rot, cap,   \
                         n - cnt);                                                                                       \
  }
  if (dtype == DJV_DTYPE_BF16) DJV_GO(bf16) else DJV_GO(float)
#undef DJV_GO
  count_launch(store == 2 && !vec ? 2 : 1);
  return check_launch("latent_rows");
}

extern "C" int djv_latent_attn(int dtype, void *out, const void *q, long long ldq, const void *kv, long long ldkv,
                               const void *tail, long long ldt, const void *gate, long long ldg, const long long *pos,
                               int B, int n, int past, int H, int dim, int rot, int dv, int window, float scale,
                               void *stream) {
  DJV_REQUIRE(dtype == DJV_DTYPE_BF16 || dtype == DJV_DTYPE_F32, "latent_attn: dtype %d", dtype);
  DJV_REQUIRE(out && q && kv && pos && (tail || rot == 0), "latent_attn: null pointer");
  DJV_REQUIRE(B >= 1 && B <= 65535 && n >= 1 && past >= 0 && H >= 1 && H <= 65535, "latent_attn: B=%d n=%d past=%d H=%d", B,
              n, past, H);
  DJV_REQUIRE(dim >= 1 && rot >= 0 && dim + rot <= 512 && dv >= 1 && dv <= 512 && window >= 1,
              "latent_attn: head sizes %d + %d / %d (up to 512), window %d", dim, rot, dv, window);
  DJV_REQUIRE(ldq >= (long long)H * (dim + rot) && ldkv >= (long long)H * (dim + dv) && ldt >= rot &&
                  (!gate || ldg >= (long long)H * dv),
              "latent_attn: a row stride is too small");
  const char *v = static_cast<const char *>(kv) + (size_t)H * dim * dtype_bytes(dtype);
  const WindowArgs a{out, q, ldq, kv, ldkv, v, ldkv, tail, ldt, rot, gate, ldg, nullptr, nullptr, nullptr, pos, B, n, H, H,
                     dim + rot, dv, 1, past, window, scale};
  return window_attn_portion(dtype, a, static_cast<cudaStream_t>(stream));
}

extern "C" size_t djv_latent_scratch_floats(int B, int H, int rank, int window) {
  if (B < 1 || H < 1 || rank < 1 || window < 1) return 0;
  return (size_t)B * H * latent_splits(B, H, window) * (rank + 2);
}

extern "C" int djv_latent_decode(int dtype, void *out, void *qc, float *scratch, size_t scratch_floats, const void *proj,
                                 long long ld, const void *uk, const void *uv, const float *norm, float eps,
                                 const float *freqs, void *ring, const void *gate, long long ldg, const long long *pos,
                                 int B, int H, int dim, int rot, int dv, int rank, int cap, int window, float scale,
                                 int stages, void *stream) {
  int rc = check_latent("latent_decode", dtype, B, 1, rank, rot, cap);
  if (rc) return rc;
  DJV_REQUIRE(out && qc && proj && uk && uv && norm && ring && pos && (freqs || rot == 0), "latent_decode: null pointer");
  DJV_REQUIRE(H >= 1 && H <= 65535 && dim >= 1 && dim <= 1024 && dv >= 1 && window >= 1,
              "latent_decode: H=%d head sizes %d / %d window=%d", H, dim, dv, window);
  DJV_REQUIRE(ld >= (long long)H * (dim + rot) + rank + rot && (!gate || ldg >= (long long)H * dv),
              "latent_decode: a row stride is too small");
  if (window > cap) window = cap;  // a ring that is shorter than the window holds the longest sequence
  const int splits = latent_splits(B, H, window);
  const size_t sums = (size_t)B * H * splits * rank, need = sums + (size_t)B * H * splits * 2;
  if (!scratch || scratch_floats < need) {
    set_error("latent_decode: scratch needs %zu floats (got %zu)", need, scratch_floats);
    return DJV_ERR_SCRATCH;
  }
  const LatentDecodeArgs a{out, qc, scratch, scratch + sums, proj, ld, uk, uv, norm, eps, freqs, ring, gate, ldg, pos, B, H,
                           dim, rot, dv, rank, cap, window, splits, scale};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool b16 = dtype == DJV_DTYPE_BF16;
  if (stages & 1) rc = b16 ? launch_query<bf16>(a, st) : launch_query<float>(a, st);
  if (rc) return rc;
  if (stages & 2) rc = b16 ? launch_attend<bf16>(a, st) : launch_attend<float>(a, st);
  if (rc) return rc;
  if (stages & 4) rc = b16 ? launch_out<bf16>(a, st) : launch_out<float>(a, st);
  return rc;
}
