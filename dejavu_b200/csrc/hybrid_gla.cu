// Gated linear attention: per head a (dk, dv) fp32 state with a decay per key channel,
//   S_t = diag(alpha_t) S_(t-1) + k_t v_t^T,   o_t = S_t^T q_t,
// followed by an RMS norm over dv and a silu gate.
//
// A portion of tokens is cut into chunks of C. With B_t[c] the sum of log alpha over the chunk up to and including t,
//   o_t = sum_c q_t[c] exp(B_t[c]) S_in[c, :]  +  sum_(s <= t) (sum_c q_t[c] k_s[c] exp(B_t[c] - B_s[c])) v_s
//   S_out[c, :] = exp(B_C[c]) S_in[c, :] + sum_s k_s[c] exp(B_C[c] - B_s[c]) v_s
// All exponents are <= 0, whatever the decays are. Three kernels: every chunk's own contribution to the state (chunks
// in parallel), a scan over the chunks that turns contributions into incoming states, every chunk's outputs (in
// parallel, norm and gate included). The kernels here do the chunks' products in fp32 on the CUDA cores, for any head
// size and both element types; the tensor-core form for bf16 is in hybrid_gla_mma.cu.
#include <cooperative_groups.h>

#include "../../include/dejavu_b200_hybrid.h"
#include "hybrid_gla.cuh"

namespace djv {

namespace cg = cooperative_groups;

// log of the decay of channel c (in 0 .. H*dk) from the low-rank activations of one token
template <typename T>
__device__ __forceinline__ float log_decay(const T *t_row, const float *a2, const float *bias, int rank, float inv_tau) {
  float z = *bias;
  for (int r = 0; r < rank; ++r) z = fmaf(to_f(t_row[r]), a2[r], z);
  return log_sigmoid_f(z) * inv_tau;
}

// sizes rounded up to whole 4x4 register tiles
__host__ __device__ __forceinline__ int up4(int v) { return (v + 3) & ~3; }

template <typename T>
__global__ void __launch_bounds__(GLA_THREADS) gla_chunk_state_kernel(GlaArgs a) {
  extern __shared__ float sm[];
  pdl_prologue();
  const int tid = threadIdx.x;
  const int ci = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const int dk = a.dk, dv = a.dv, dkp = up4(dk), dvp = up4(dv);
  const int t0 = ci * a.C, cl = min(a.C, a.n - t0);
  float *ks = sm, *vs = ks + a.C * dkp, *bs = vs + a.C * dvp;  // [C][dkp], [C][dvp], [C][dkp]
  const T *rows = static_cast<const T *>(a.proj) + ((size_t)b * a.n + t0) * a.ld;
  const int koff = a.H * dk + h * dk, voff = 2 * a.H * dk + h * dv, toff = 2 * a.H * dk + 2 * a.H * dv;
  for (int i = tid; i < cl * dk; i += GLA_THREADS) {
    const int t = i / dk, c = i % dk;
    bs[t * dkp + c] = log_decay(rows + (size_t)t * a.ld + toff, a.a2 + (size_t)(h * dk + c) * a.rank,
                                a.a2_bias + h * dk + c, a.rank, a.inv_tau);
  }
  for (int i = tid; i < cl * dvp; i += GLA_THREADS) {
    const int t = i / dvp, j = i % dvp;
    vs[i] = j < dv ? to_f(rows[(size_t)t * a.ld + voff + j]) : 0.f;
  }
  __syncthreads();
  for (int c = tid; c < dkp; c += GLA_THREADS) {
    float run = 0.f;
    if (c < dk) {
      for (int t = 0; t < cl; ++t) {
        run += bs[t * dkp + c];
        bs[t * dkp + c] = run;
        a.cum[(((size_t)b * a.n + t0 + t) * a.H + h) * dk + c] = run;
      }
      a.decay[(((size_t)b * a.H + h) * a.nc + ci) * dk + c] = run;
    }
    for (int t = 0; t < cl; ++t)
      ks[t * dkp + c] = c < dk ? to_f(rows[(size_t)t * a.ld + koff + c]) * expf(run - bs[t * dkp + c]) : 0.f;
  }
  __syncthreads();
  float *U = a.contrib + (((size_t)b * a.H + h) * a.nc + ci) * (size_t)dk * dv;
  const int tk = dkp / 4, tv = dvp / 4;
  for (int tile = tid; tile < tk * tv; tile += GLA_THREADS) {
    const int c0 = tile / tv * 4, j0 = tile % tv * 4;
    float acc[4][4] = {};
    for (int t = 0; t < cl; ++t) {
      const float4 k4 = *reinterpret_cast<const float4 *>(ks + t * dkp + c0);
      const float4 v4 = *reinterpret_cast<const float4 *>(vs + t * dvp + j0);
      const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, vv[4] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
      for (int x = 0; x < 4; ++x)
#pragma unroll
        for (int y = 0; y < 4; ++y) acc[x][y] = fmaf(kk[x], vv[y], acc[x][y]);
    }
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
      for (int y = 0; y < 4; ++y)
        if (c0 + x < dk && j0 + y < dv) U[(size_t)(c0 + x) * dv + j0 + y] = acc[x][y];
  }
}

// contributions -> incoming states, V neighbouring state elements of one row per thread, chunks in order
template <int V>
__global__ void __launch_bounds__(GLA_THREADS) gla_state_scan_kernel(GlaArgs a) {
  pdl_prologue();
  const int per = a.dk * a.dv;
  const int e = (blockIdx.x * GLA_THREADS + threadIdx.x) * V;
  const int h = blockIdx.y, b = blockIdx.z;
  if (e >= per) return;
  const size_t bh = (size_t)b * a.H + h;
  auto get = [](const float *p, float (&v)[V]) {
    if (V == 2) {
      const float2 t = *reinterpret_cast<const float2 *>(p);
      v[0] = t.x; v[1 % V] = t.y;
    } else {
      v[0] = *p;
    }
  };
  auto put = [](float *p, const float (&v)[V]) {
    if (V == 2)
      *reinterpret_cast<float2 *>(p) = make_float2(v[0], v[1 % V]);
    else
      *p = v[0];
  };
  float s[V];
#pragma unroll
  for (int v = 0; v < V; ++v) s[v] = 0.f;
  if (a.pos[b] != 0) get(a.state + bh * per + e, s);
  float *U = a.contrib + bh * a.nc * per + e;
  const float *D = a.decay + bh * a.nc * a.dk + e / a.dv;
  constexpr int CH = 8;  // chunks whose loads are in flight together
  int c0 = 0;
  for (; c0 + CH <= a.nc; c0 += CH, U += (size_t)CH * per, D += CH * a.dk) {
    float u[CH][V], d[CH];
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      get(U + (size_t)c * per, u[c]);
      d[c] = D[c * a.dk];
    }
#pragma unroll
    for (int c = 0; c < CH; ++c) {
      put(U + (size_t)c * per, s);
      const float f = expf(d[c]);
#pragma unroll
      for (int v = 0; v < V; ++v) s[v] = fmaf(f, s[v], u[c][v]);
    }
  }
  for (; c0 < a.nc; ++c0, U += per, D += a.dk) {
    float u[V];
    get(U, u);
    put(U, s);
    const float f = expf(*D);
#pragma unroll
    for (int v = 0; v < V; ++v) s[v] = fmaf(f, s[v], u[v]);
  }
  put(a.state + bh * per + e, s);
}

template <typename T>
__global__ void __launch_bounds__(GLA_THREADS) gla_chunk_out_kernel(GlaArgs a) {
  extern __shared__ float sm[];
  pdl_prologue();
  const int tid = threadIdx.x, lane = tid % WARP, warp = tid / WARP;
  const int ci = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const int dk = a.dk, dv = a.dv, C = a.C, dvp = up4(dv), kp = dk | 1;
  const int t0 = ci * C, cl = min(C, a.n - t0);
  float *qs = sm, *ks = qs + C * kp, *bs = ks + C * kp, *A = bs + C * kp;  // [C][kp] x3, [C][C]
  float *vs = A + C * C;                                                   // [C][dvp]; o afterwards
  vs = sm + up4((int)(vs - sm));
  const T *rows = static_cast<const T *>(a.proj) + ((size_t)b * a.n + t0) * a.ld;
  const int qoff = h * dk, koff = a.H * dk + h * dk, voff = 2 * a.H * dk + h * dv, goff = voff + a.H * dv;
  for (int i = tid; i < cl * dk; i += GLA_THREADS) {
    const int t = i / dk, c = i % dk;
    const T *r = rows + (size_t)t * a.ld;
    qs[t * kp + c] = to_f(r[qoff + c]) * a.scale;
    ks[t * kp + c] = to_f(r[koff + c]);
    bs[t * kp + c] = a.cum[(((size_t)b * a.n + t0 + t) * a.H + h) * dk + c];
  }
  for (int i = tid; i < cl * dvp; i += GLA_THREADS) {
    const int t = i / dvp, j = i % dvp;
    vs[i] = j < dv ? to_f(rows[(size_t)t * a.ld + voff + j]) : 0.f;
  }
  __syncthreads();
  for (int i = tid; i < cl * cl; i += GLA_THREADS) {
    const int t = i / cl, s = i % cl;
    float acc = 0.f;
    if (s <= t)
      for (int c = 0; c < dk; ++c)
        acc = fmaf(qs[t * kp + c] * ks[s * kp + c], expf(bs[t * kp + c] - bs[s * kp + c]), acc);
    A[t * C + s] = acc;
  }
  __syncthreads();
  for (int i = tid; i < cl * dk; i += GLA_THREADS) {
    const int t = i / dk, c = i % dk;
    qs[t * kp + c] *= expf(bs[t * kp + c]);
  }
  __syncthreads();
  const float *S = a.contrib + (((size_t)b * a.H + h) * a.nc + ci) * (size_t)dk * dv;
  float *os = ks;  // the keys and sums are not needed any more: outputs [C][dvp] go over them when they fit
  const bool fits = C * dvp <= 2 * C * kp;
  if (!fits) os = vs + C * dvp;
  const int tt = (cl + 3) / 4, tv = dvp / 4;
  for (int tile = tid; tile < tt * tv; tile += GLA_THREADS) {
    const int r0 = tile / tv * 4, j0 = tile % tv * 4;
    float acc[4][4] = {};
    for (int c = 0; c < dk; ++c) {
      float sv[4];
#pragma unroll
      for (int y = 0; y < 4; ++y) sv[y] = j0 + y < dv ? S[(size_t)c * dv + j0 + y] : 0.f;
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const float q = r0 + x < cl ? qs[(r0 + x) * kp + c] : 0.f;
#pragma unroll
        for (int y = 0; y < 4; ++y) acc[x][y] = fmaf(q, sv[y], acc[x][y]);
      }
    }
    for (int s = 0; s < min(cl, r0 + 4); ++s) {
      const float4 v4 = *reinterpret_cast<const float4 *>(vs + s * dvp + j0);
      const float vv[4] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
      for (int x = 0; x < 4; ++x) {
        const float p = r0 + x < cl ? A[(r0 + x) * C + s] : 0.f;
#pragma unroll
        for (int y = 0; y < 4; ++y) acc[x][y] = fmaf(p, vv[y], acc[x][y]);
      }
    }
#pragma unroll
    for (int x = 0; x < 4; ++x)
#pragma unroll
      for (int y = 0; y < 4; ++y)
        if (r0 + x < cl) os[(r0 + x) * dvp + j0 + y] = acc[x][y];
  }
  __syncthreads();
  for (int t = warp; t < cl; t += GLA_THREADS / WARP) {
    float ss = 0.f;
    for (int j = lane; j < dv; j += WARP) ss = fmaf(os[t * dvp + j], os[t * dvp + j], ss);
    ss = warp_sum(ss);
    const float r = 1.f / sqrtf(ss / (float)dv + a.eps);
    const T *row = rows + (size_t)t * a.ld;
    T *out = static_cast<T *>(a.out) + (((size_t)b * a.n + t0 + t) * a.H + h) * dv;
    for (int j = lane; j < dv; j += WARP) {
      const float g = to_f(row[goff + j]);
      out[j] = from_f<T>(os[t * dvp + j] * r * a.norm[j] * (g * sigmoid_f(g)));
    }
  }
}

// ---- decode: one token per sequence ------------------------------------------------------------------------------
// grid (column blocks, H, B), a cluster over the column blocks of a head (the norm needs all of dv). A block reads,
// updates and writes its (dk, columns) part of the state once; the first batch of state loads is in flight while the
// decays are computed, and the decay weights are fetched before the kernel waits for its predecessor.
constexpr int GD_THREADS = 128;
constexpr int GD_MAX_BLOCKS = 8;
constexpr int GD_ROWS = 8;  // state rows of a thread per batch of loads

template <typename T, int V>
__global__ void __launch_bounds__(GD_THREADS) gla_decode_kernel(GlaArgs a, int cols) {
  extern __shared__ float sm[];
  __shared__ float red[GD_THREADS / WARP];
  __shared__ float ss_all[GD_MAX_BLOCKS];
  const int tid = threadIdx.x;
  const int cb = blockIdx.x, h = blockIdx.y, b = blockIdx.z, dk = a.dk, dv = a.dv, nb = gridDim.x;
  const int j0 = cb * cols, jn = max(0, min(cols, dv - j0));
  const int wp = a.rank + 1;
  float *q = sm, *k = q + dk, *al = k + dk, *w = al + dk, *osum = w + dk * wp;  // osum: [row groups][cols]
  cg::cluster_group cluster = cg::this_cluster();
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  if (nb > 1) cluster.barrier_arrive();  // (waited for before the first access to another block's memory)
  for (int i = tid; i < dk * a.rank; i += GD_THREADS)
    w[i / a.rank * wp + i % a.rank] = a.a2[(size_t)h * dk * a.rank + i];
  asm volatile("griddepcontrol.wait;" ::: "memory");
  const T *row = static_cast<const T *>(a.proj) + (size_t)b * a.ld;
  const T *v = row + 2 * a.H * dk + h * dv + j0, *gate = v + a.H * dv;
  const T *tr = row + 2 * a.H * dk + 2 * a.H * dv;
  const bool fresh = a.pos[b] == 0;
  float *S = a.state + ((size_t)b * a.H + h) * dk * dv + j0;
  const int groups = jn / V;                                  // column groups (V divides cols and dv)
  const int rows = max(1, GD_THREADS / max(1, groups));       // row groups
  const int cg0 = tid % max(1, groups) * V, r = tid / max(1, groups);
  const bool mine = r < rows && groups > 0;
  float st[GD_ROWS][V];
  auto fetch = [&](int c0) {
#pragma unroll
    for (int x = 0; x < GD_ROWS; ++x) {
      const int c = c0 + x * rows;
      const bool ok = mine && c < dk && !fresh;
      const float *p = S + (size_t)c * dv + cg0;
      if (V == 4) {
        float4 t = make_float4(0.f, 0.f, 0.f, 0.f);
        if (ok) t = *reinterpret_cast<const float4 *>(p);
        st[x][0] = t.x; st[x][1 % V] = t.y; st[x][2 % V] = t.z; st[x][3 % V] = t.w;
      } else {
        st[x][0] = ok ? p[0] : 0.f;
      }
    }
  };
  fetch(r);
  __syncthreads();  // w[] is complete
  for (int c = tid; c < dk; c += GD_THREADS) {
    q[c] = to_f(row[h * dk + c]) * a.scale;
    k[c] = to_f(row[a.H * dk + h * dk + c]);
    al[c] = expf(log_decay(tr, w + c * wp, a.a2_bias + h * dk + c, a.rank, a.inv_tau));
  }
  __syncthreads();
  float vv[V], acc[V];
#pragma unroll
  for (int e = 0; e < V; ++e) {
    vv[e] = mine ? to_f(v[cg0 + e]) : 0.f;
    acc[e] = 0.f;
  }
  for (int c0 = r; c0 < dk; c0 += GD_ROWS * rows) {
    if (c0 != r) fetch(c0);
#pragma unroll
    for (int x = 0; x < GD_ROWS; ++x) {
      const int c = c0 + x * rows;
      if (!mine || c >= dk) continue;
      float *p = S + (size_t)c * dv + cg0;
#pragma unroll
      for (int e = 0; e < V; ++e) {
        st[x][e] = fmaf(k[c], vv[e], al[c] * st[x][e]);
        acc[e] = fmaf(q[c], st[x][e], acc[e]);
      }
      if (V == 4)
        *reinterpret_cast<float4 *>(p) = make_float4(st[x][0], st[x][1 % V], st[x][2 % V], st[x][3 % V]);
      else
        p[0] = st[x][0];
    }
  }
  if (mine) {
#pragma unroll
    for (int e = 0; e < V; ++e) osum[r * cols + cg0 + e] = acc[e];
  }
  __syncthreads();
  float ss = 0.f;
  for (int j = tid; j < jn; j += GD_THREADS) {
    float o = 0.f;
    for (int x = 0; x < rows; ++x) o += osum[x * cols + j];
    osum[j] = o;  // row group 0's slot of the same column, read by this thread only
    ss = fmaf(o, o, ss);
  }
  ss = warp_sum(ss);
  if (tid % WARP == 0) red[tid / WARP] = ss;
  __syncthreads();
  float tot = 0.f;
#pragma unroll
  for (int x = 0; x < GD_THREADS / WARP; ++x) tot += red[x];
  if (nb > 1) {
    cluster.barrier_wait();
    if (tid < nb) cluster.map_shared_rank(ss_all, tid)[cb] = tot;  // this block's sum to every block
    cluster.sync();
    tot = 0.f;
    for (int x = 0; x < nb; ++x) tot += ss_all[x];
  }
  const float rn = 1.f / sqrtf(tot / (float)dv + a.eps);
  T *out = static_cast<T *>(a.out) + ((size_t)b * a.H + h) * dv + j0;
  for (int j = tid; j < jn; j += GD_THREADS) {
    const float g = to_f(gate[j]);
    out[j] = from_f<T>(osum[j] * rn * a.norm[j0 + j] * (g * sigmoid_f(g)));
  }
}

// ---- host ----------------------------------------------------------------------------------------------------------
static size_t state_smem(int C, int dk, int dv) { return 4 * (size_t)C * (2 * up4(dk) + up4(dv)); }
static size_t out_smem(int C, int dk, int dv) {
  const int kp = dk | 1, dvp = up4(dv);
  size_t f = (size_t)3 * C * kp + (size_t)C * C + 4 + (size_t)C * dvp;
  if (C * dvp > 2 * C * kp) f += (size_t)C * dvp;
  return 4 * f;
}
constexpr size_t GLA_SMEM = 220 * 1024;
// chunk length: as long as both kernels' tiles fit into shared memory, 0 if the heads are too large
static int chunk_len(int dk, int dv) {
  for (int C = 64; C >= 8; C /= 2)
    if (state_smem(C, dk, dv) <= GLA_SMEM && out_smem(C, dk, dv) <= GLA_SMEM) return C;
  return 0;
}
static size_t al256(size_t v) { return (v + 255) / 256 * 256; }

// the tensor-core chunk kernels also need rows that 16-byte copies can read
static bool use_mma(int dtype, const GlaArgs &a) {
  return gla_mma_supported(dtype, a.dk, a.dv) && a.ld % 8 == 0 && aligned16(a.proj) && aligned16(a.out) &&
         aligned16(a.norm);
}

template <typename T>
static int launch_prefill(const GlaArgs &a, bool mma, cudaStream_t st) {
  const size_t s1 = state_smem(a.C, a.dk, a.dv), s3 = out_smem(a.C, a.dk, a.dv);
  const dim3 grid(a.nc, a.H, a.B);
  int rc = DJV_OK;
  if (mma) {
    rc = gla_mma_chunk_state(a, st);
  } else {
    cudaFuncSetAttribute(gla_chunk_state_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)GLA_SMEM);
    djv::launch_kernel(gla_chunk_state_kernel<T>, grid, dim3(GLA_THREADS), s1, st, a);
    count_launch();
  }
  if (rc) return rc;
  if (a.dv % 2 == 0 && aligned16(a.state))
    djv::launch_kernel(gla_state_scan_kernel<2>, dim3(ceil_div(a.dk * a.dv, 2 * GLA_THREADS), a.H, a.B),
                       dim3(GLA_THREADS), 0, st, a);
  else
    djv::launch_kernel(gla_state_scan_kernel<1>, dim3(ceil_div(a.dk * a.dv, GLA_THREADS), a.H, a.B), dim3(GLA_THREADS),
                       0, st, a);
  count_launch();
  if (mma) return gla_mma_chunk_out(a, st);
  cudaFuncSetAttribute(gla_chunk_out_kernel<T>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)GLA_SMEM);
  djv::launch_kernel(gla_chunk_out_kernel<T>, grid, dim3(GLA_THREADS), s3, st, a);
  count_launch();
  return check_launch("gla_prefill");
}

template <typename T>
static int launch_gla_decode(const GlaArgs &a, cudaStream_t st) {
  const bool vec = a.dv % 4 == 0 && aligned16(a.state);
  const int V = vec ? 4 : 1;
  int nb = 1;  // column blocks: at least 16 columns each
  while (nb < GD_MAX_BLOCKS && a.dv >= 32 * nb) nb *= 2;
  const int cols = ceil_div(ceil_div(a.dv, nb), V) * V;
  nb = ceil_div(a.dv, cols);
  const int rows = GD_THREADS / (cols / V) > 1 ? GD_THREADS / (cols / V) : 1;
  // the last block may have fewer columns, hence more row groups of them: bounded by threads * V outputs
  size_t osum = (size_t)rows * cols;
  const int last = a.dv - (nb - 1) * cols;
  const int last_rows = GD_THREADS / (last / V > 0 ? last / V : 1) > 1 ? GD_THREADS / (last / V > 0 ? last / V : 1) : 1;
  if ((size_t)last_rows * cols > osum) osum = (size_t)last_rows * cols;
  const size_t smem = 4 * ((size_t)a.dk * (3 + a.rank + 1) + osum);
  DJV_REQUIRE(smem <= 200 * 1024, "gla_decode: head sizes %d / %d, rank %d are too large", a.dk, a.dv, a.rank);
  const dim3 grid(nb, a.H, a.B), cluster(nb, 1, 1);
  if (vec) {
    cudaFuncSetAttribute(gla_decode_kernel<T, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    djv::launch_kernel_cluster(gla_decode_kernel<T, 4>, grid, dim3(GD_THREADS), smem, st, cluster, a, cols);
  } else {
    cudaFuncSetAttribute(gla_decode_kernel<T, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    djv::launch_kernel_cluster(gla_decode_kernel<T, 1>, grid, dim3(GD_THREADS), smem, st, cluster, a, cols);
  }
  count_launch();
  return check_launch("gla_decode");
}

}  // namespace djv

using namespace djv;

static int check_gla(const char *op, int dtype, const GlaArgs &a) {
  DJV_REQUIRE(dtype == DJV_DTYPE_BF16 || dtype == DJV_DTYPE_F32, "%s: dtype %d", op, dtype);
  DJV_REQUIRE(a.out && a.proj && a.a2 && a.a2_bias && a.norm && a.state && a.pos, "%s: null pointer", op);
  DJV_REQUIRE(a.B >= 1 && a.B <= 65535 && a.n >= 1 && a.H >= 1 && a.H <= 65535, "%s: B=%d n=%d H=%d", op, a.B, a.n, a.H);
  DJV_REQUIRE(a.dk >= 1 && a.dv >= 1 && a.dk <= 512 && a.dv <= 512 && a.rank >= 1, "%s: head sizes %d / %d, rank %d", op,
              a.dk, a.dv, a.rank);
  DJV_REQUIRE(a.ld >= 2ll * a.H * (a.dk + a.dv) + a.rank, "%s: row stride %lld is too small", op, a.ld);
  return DJV_OK;
}

extern "C" size_t djv_gla_scratch_bytes(int dtype, int B, int n, int H, int dk, int dv) {
  if (B < 1 || n < 1 || H < 1 || dk < 1 || dv < 1) return 0;
  int C = chunk_len(dk, dv);
  if (gla_mma_supported(dtype, dk, dv) && (C == 0 || C > GLA_MMA_CHUNK)) C = GLA_MMA_CHUNK;
  if (C == 0) return 0;
  const size_t nc = ceil_div(n, C), bh = (size_t)B * H;
  return al256(bh * nc * dk * dv * 4) + al256(bh * nc * dk * 4) + al256(bh * n * dk * 4);
}

extern "C" int djv_gla_prefill(int dtype, void *out, const void *proj, long long ld, const float *a2,
                               const float *a2_bias, int rank, float inv_tau, const float *norm, float eps, float scale,
                               float *state, const long long *pos, int B, int n, int H, int dk, int dv, void *scratch,
                               size_t scratch_bytes, void *stream) {
  GlaArgs a{out, proj, ld, a2, a2_bias, norm, inv_tau, eps, scale, state, pos, B, n, H, dk, dv, rank, 0, 0, nullptr,
            nullptr, nullptr};
  int rc = check_gla("gla_prefill", dtype, a);
  if (rc) return rc;
  const bool mma = use_mma(dtype, a);
  a.C = mma ? GLA_MMA_CHUNK : chunk_len(dk, dv);
  if (a.C == 0) {
    set_error("gla_prefill: head sizes %d / %d are too large", dk, dv);
    return DJV_ERR_UNSUPPORTED;
  }
  a.nc = ceil_div(n, a.C);
  const size_t need = djv_gla_scratch_bytes(dtype, B, n, H, dk, dv);
  if (!scratch || scratch_bytes < need || !aligned16(scratch)) {
    set_error("gla_prefill: scratch needs %zu bytes (got %zu)", need, scratch_bytes);
    return DJV_ERR_SCRATCH;
  }
  char *p = static_cast<char *>(scratch);
  const size_t bh = (size_t)B * H;
  a.contrib = reinterpret_cast<float *>(p);
  p += al256(bh * a.nc * dk * dv * 4);
  a.decay = reinterpret_cast<float *>(p);
  p += al256(bh * a.nc * dk * 4);
  a.cum = reinterpret_cast<float *>(p);
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == DJV_DTYPE_BF16 ? launch_prefill<bf16>(a, mma, st) : launch_prefill<float>(a, false, st);
}

extern "C" int djv_gla_decode(int dtype, void *out, const void *proj, long long ld, const float *a2,
                              const float *a2_bias, int rank, float inv_tau, const float *norm, float eps, float scale,
                              float *state, const long long *pos, int B, int H, int dk, int dv, void *stream) {
  const GlaArgs a{out, proj, ld, a2, a2_bias, norm, inv_tau, eps, scale, state, pos, B, 1, H, dk, dv, rank, 0, 0,
                  nullptr, nullptr, nullptr};
  int rc = check_gla("gla_decode", dtype, a);
  if (rc) return rc;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == DJV_DTYPE_BF16 ? launch_gla_decode<bf16>(a, st) : launch_gla_decode<float>(a, st);
}
