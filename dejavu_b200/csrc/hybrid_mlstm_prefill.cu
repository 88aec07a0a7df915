// The chunk kernels of the matrix memory on the 5th-generation tensor cores (bf16 projections), chunks of 128 tokens.
//
// State: U (TMEM, channels x values) = (w K)^T V, w_s = e^(a_s - max a). The weighted keys are fp32 numbers and enter as two
// bf16 terms, hi + lo.
// Outputs: S = Q K^T (TMEM); P_ts = S_ts e^(a_s - M_t) for s <= t goes back to TMEM over S, as hi + lo; O (TMEM) = Q S_in, S_in
// in hi + lo, scaled by e^(m_in - M_t) row by row, then += P_hi V + P_lo V. The denominator takes the fp32 sums of P and
// q . n_in. Norm and gate run on the way out. The incoming state streams through two buffers of 64 channels; V takes the one
// that is free first, the output gates the other. A block has 256 threads, two per row of TMEM, and up to 256 value
// columns; wider heads are a cluster of blocks that exchange their sums of squares.
#include <cooperative_groups.h>

#include "../../include/dejavu_b200_routed.h"
#include "hybrid_mlstm.cuh"
#include "tcgen05.cuh"

namespace djv {

namespace cg = cooperative_groups;

constexpr int MT_C = MLSTM_TC_CHUNK;             // tokens per chunk, rows of every tile
constexpr uint32_t MT_BLOCK = MT_C * 128;        // bytes of a 64-column block of such a tile
constexpr int MT_MAX_TILES = 8;                  // value tiles of a head (blocks of a cluster)
constexpr double LOG2E = 1.4426950408889634;

__device__ unsigned g_mlstm_timeouts;  // bounded waits that ran out (never, in a healthy run)

__device__ __forceinline__ float exp2_fast(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// rows of `cols` elements (stride ld) into NB 64-column blocks of ROWS swizzled rows, zeros outside
template <int NB, int ROWS>
__device__ __forceinline__ void load_tile(uint32_t dst, const bf16 *src, long long ld, int rows, int cols) {
#pragma unroll 4
  for (int i = threadIdx.x; i < ROWS * NB * 8; i += ML_THREADS) {
    const int r = i / (NB * 8), ch = i - r * (NB * 8);
    const bool ok = r < rows && ch * 8 < cols;
    cp_async16_zfill(dst + sw128_offset(ROWS, r, ch), ok ? src + (long long)r * ld + ch * 8 : src, ok ? 16 : 0);
  }
}

// two floats -> packed bf16 pairs hi (upper halves) and lo (what they leave out, rounded)
__device__ __forceinline__ void split_pair(float x, float y, uint32_t &hi, uint32_t &lo) {
  hi = __byte_perm(__float_as_uint(x), __float_as_uint(y), 0x7632);
  lo = pack_bf16(x - __uint_as_float(__float_as_uint(x) & 0xffff0000u), y - __uint_as_float(__float_as_uint(y) & 0xffff0000u));
}

// ---- gates of all chunks, a warp each ----------------------------------------------------------------------------------
constexpr int MG_WARPS = 4;
__global__ void __launch_bounds__(MG_WARPS * WARP) mlstm_tc_gates_kernel(MlstmArgs a) {
  __shared__ float2 as[MG_WARPS][MT_C];
  __shared__ double run[MG_WARPS][MT_C], sum[MG_WARPS][MT_C];
  pdl_prologue();
  const int warp = threadIdx.x / WARP, lane = threadIdx.x % WARP, ci = blockIdx.x * MG_WARPS + warp;
  const int h = blockIdx.y, b = blockIdx.z;
  if (ci >= a.nc) return;
  double total, top;
  chunk_gates<MT_C / WARP>(a, b, h, ci * MT_C, min(MT_C, a.n - ci * MT_C), as[warp], run[warp], sum[warp], total, top);
  __syncwarp();
  const size_t at = ((size_t)b * a.H + h) * a.nc + ci;
  for (int t = lane; t < MT_C; t += WARP) {
    a.g_a[at * MT_C + t] = as[warp][t];
    a.g_run[at * MT_C + t] = run[warp][t];
    a.g_sum[at * MT_C + t] = sum[warp][t];
  }
  if (lane == 0) {
    a.chunk[at * 3] = total;
    a.chunk[at * 3 + 1] = top;
  }
}

// ---- a chunk's own contribution to the state -----------------------------------------------------------------------
template <int KB, int VB>  // 64-column blocks: keys (2 or 4: M comes in 128 channels), values
__global__ void __launch_bounds__(ML_THREADS, KB > 2 ? 1 : 2) mlstm_tc_chunk_state_kernel(MlstmArgs a, int nvt) {
  extern __shared__ unsigned char smem_raw[];
  __shared__ __align__(8) uint64_t bar;
  __shared__ uint32_t tmem_slot;
  constexpr int PER = KB * 8, STEP = ML_THREADS / PER;  // chunks of 8 channels in a row, rows at a time
  __shared__ float wt[MT_C], nsum[STEP][KB * 64];
  constexpr uint32_t COLS = KB > 2 ? 256 : (VB > 1 ? 128 : 64);
  constexpr int MT = KB / 2;
  const int tid = threadIdx.x, warp = tid / WARP;
  const int vt = blockIdx.x % nvt, ci = blockIdx.x / nvt, h = blockIdx.y, b = blockIdx.z;
  const int dk = a.dk, dv = a.dv, v0 = vt * VB * 64, vn = min(VB * 64, dv - v0);
  const int t0 = ci * MT_C, cl = min(MT_C, a.n - t0);
  unsigned char *base = reinterpret_cast<unsigned char *>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const uint32_t hi_sm = smem_u32(base), lo_sm = hi_sm + KB * MT_BLOCK, v_sm = lo_sm + KB * MT_BLOCK;
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");
  if (tid == 0) {
    mbar_init(&bar, 1);
    mbar_fence_init();
  }
  const bf16 *rows = static_cast<const bf16 *>(a.proj) + ((size_t)b * a.n + t0) * a.ld;
  load_tile<KB, MT_C>(hi_sm, rows + (size_t)(a.H + h) * dk, a.ld, cl, dk);
  cp_async_commit();
  load_tile<VB, MT_C>(v_sm, rows + (size_t)2 * a.H * dk + (size_t)h * dv + v0, a.ld, cl, vn);
  cp_async_commit();
  const size_t at = ((size_t)b * a.H + h) * a.nc + ci;
  __syncwarp();
  if (warp == 0) tmem_alloc(&tmem_slot, COLS);
  if (tid < MT_C) wt[tid] = exp_diff(a.g_a[at * MT_C + tid], split_double(a.chunk[at * 3 + 1]));
  cp_async_wait<1>();
  __syncthreads();
  {  // weighted keys, split in place; a thread keeps its chunk of 8 channels over the rows and sums them for n
    const int ch = tid % PER;
    float s[8] = {};
    for (int r = tid / PER; r < MT_C; r += STEP) {
      uint4 *p = reinterpret_cast<uint4 *>(base + sw128_offset(MT_C, r, ch));
      float f[8];
      unpack_chunk<bf16>(*p, f);
      uint4 hi, lo;
      uint32_t *hp = &hi.x, *lp = &lo.x;
      const float w = wt[r];
#pragma unroll
      for (int e = 0; e < 8; e += 2) {
        const float x = f[e] * w, y = f[e + 1] * w;
        s[e] += x;
        s[e + 1] += y;
        split_pair(x, y, hp[e / 2], lp[e / 2]);
      }
      *p = hi;
      *reinterpret_cast<uint4 *>(base + KB * MT_BLOCK + sw128_offset(MT_C, r, ch)) = lo;
    }
#pragma unroll
    for (int e = 0; e < 8; ++e) nsum[tid / PER][ch * 8 + e] = s[e];
  }
  cp_async_wait<0>();
  fence_proxy_async_smem();
  __syncthreads();
  tmem_fence_after();
  const uint32_t tm = tmem_slot;
  const int np = (vn + 15) / 16 * 16;
  if (tid == 0) {
    const uint32_t idesc = mma_idesc(128, np, true, true);
    const uint64_t vd = desc_mn_major(v_sm, MT_C, 0);
#pragma unroll
    for (int m = 0; m < MT; ++m) {
      if (m * 128 >= dk) continue;
#pragma unroll
      for (int part = 0; part < 2; ++part) {
        const uint64_t kd = desc_mn_major((part ? lo_sm : hi_sm) + m * 2 * MT_BLOCK, MT_C, 0);
#pragma unroll
        for (int k = 0; k < MT_C / 16; ++k) mma_ss(tm + m * 128, kd + (uint64_t)(k * 128), vd + (uint64_t)(k * 128), idesc, part + k > 0);
      }
    }
    mma_commit(&bar);
  }
  float *U = a.contrib + at * mlstm_contrib_stride(dk, dv);
  if (vt == 0)
    for (int c = tid; c < dk; c += ML_THREADS) {
      float s = 0.f;
#pragma unroll
      for (int x = 0; x < STEP; ++x) s += nsum[x][c];
      U[(size_t)dk * dv + c] = s;
    }
  const bool dead = !mbar_wait(&bar, 0);
  __syncwarp();
  tmem_fence_after();
  const uint32_t lane_base = (uint32_t)(warp % 4 * 32) << 16;
  const int half = tid / 128;
#pragma unroll
  for (int m = 0; m < MT; ++m) {
    const int c = m * 128 + tid % 128;
    float *dst = U + (size_t)c * dv + v0;
    if (m * 128 < dk) {
      for (int q = half * 16; q < np; q += 32) {
        uint32_t o[16];
        tmem_ld16(o, tm + m * 128 + lane_base + q);
        tmem_wait_ld();
        if (c < dk) {
#pragma unroll
          for (int e = 0; e < 16; e += 4)
            if (q + e < vn)  // (dv % 8 == 0)
              *reinterpret_cast<float4 *>(dst + q + e) =
                  make_float4(__uint_as_float(o[e]), __uint_as_float(o[e + 1]), __uint_as_float(o[e + 2]), __uint_as_float(o[e + 3]));
        }
        __syncwarp();
      }
    }
  }
  if (dead && tid == 0) atomicAdd(&g_mlstm_timeouts, 1u);
  tmem_fence_before();
  __syncthreads();
  if (warp == 0) tmem_dealloc(tm, COLS);
}

// ---- a chunk's outputs -----------------------------------------------------------------------------------------------
template <int KB, int VB>
__global__ void __launch_bounds__(ML_THREADS, VB > 2 ? 1 : 2) mlstm_tc_chunk_out_kernel(MlstmArgs a) {
  extern __shared__ unsigned char smem_raw[];
  __shared__ __align__(8) uint64_t bar_s, bar_o, bar_buf[2];
  __shared__ uint32_t tmem_slot;
  __shared__ float2 as[MT_C], mt[MT_C];  // in units of log 2
  __shared__ float w_in[MT_C], floor_s[MT_C], exch[2][MT_C], ssq[MT_MAX_TILES][MT_C], n_in[KB * 64], norm_s[VB * 64];
  constexpr uint32_t COLS = VB > 2 ? 512 : 256;
  constexpr uint32_t SLICE = 64 * 128;            // bytes of a 64-column block of 64 channels
  constexpr uint32_t BUF = 2 * VB * SLICE;        // hi and lo of 64 channels; or 128 rows of V
  const int tid = threadIdx.x, warp = tid / WARP;
  const int half = tid / MT_C, r = tid % MT_C;
  const int vt = blockIdx.x, nvt = gridDim.x, ci = blockIdx.y, h = blockIdx.z % a.H, b = blockIdx.z / a.H;
  const int dk = a.dk, dv = a.dv, v0 = vt * VB * 64, vn = min(VB * 64, dv - v0);
  const int t0 = ci * MT_C, cl = min(MT_C, a.n - t0);
  unsigned char *base = reinterpret_cast<unsigned char *>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  const uint32_t q_sm = smem_u32(base), k_sm = q_sm + KB * MT_BLOCK, buf_sm = k_sm + KB * MT_BLOCK;
  cg::cluster_group cluster = cg::this_cluster();
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  if (nvt > 1) cluster.barrier_arrive();  // (waited for before the first access to another block's memory)
  asm volatile("griddepcontrol.wait;" ::: "memory");
  if (tid == 0) {
    mbar_init(&bar_s, 1);
    mbar_init(&bar_o, 1);
    mbar_init(&bar_buf[0], 1);
    mbar_init(&bar_buf[1], 1);
    mbar_fence_init();
  }
  const bf16 *rows = static_cast<const bf16 *>(a.proj) + ((size_t)b * a.n + t0) * a.ld;
  const bf16 *v_rows = rows + (size_t)2 * a.H * dk + (size_t)h * dv + v0, *gate = v_rows + (size_t)a.H * dv;
  const size_t at = ((size_t)b * a.H + h) * a.nc + ci;
  load_tile<KB, MT_C>(q_sm, rows + (size_t)h * dk, a.ld, cl, dk);
  load_tile<KB, MT_C>(k_sm, rows + (size_t)(a.H + h) * dk, a.ld, cl, dk);
  cp_async_commit();
  auto slice = [&](int s) {  // 64 channels of the incoming state
    const size_t off = at * dk * dv + (size_t)s * 64 * dv + v0;
    const uint32_t dst = buf_sm + (s & 1) * BUF;
    load_tile<VB, 64>(dst, a.s_hi + off, dv, dk - s * 64, vn);
    load_tile<VB, 64>(dst + VB * SLICE, a.s_lo + off, dv, dk - s * 64, vn);
    cp_async_commit();
  };
  slice(0);
  if (KB > 1) slice(1);
  __syncwarp();
  if (warp == 0) tmem_alloc(&tmem_slot, COLS);
  if (tid < MT_C) {
    const double m0 = a.chunk[at * 3 + 2], M = fmax(a.g_run[at * MT_C + tid], m0);
    const float2 x = a.g_a[at * MT_C + tid];
    mt[tid] = split_double(M * LOG2E);
    as[tid] = split_double(((double)x.x + (double)x.y) * LOG2E);
    w_in[tid] = expf((float)(m0 - M)) * a.scale;
    floor_s[tid] = expf((float)-(a.g_sum[at * MT_C + tid] + M));
  } else {
    const float *N = a.contrib + at * mlstm_contrib_stride(dk, dv) + (size_t)dk * dv;
    for (int c = tid - MT_C; c < KB * 64; c += ML_THREADS - MT_C) n_in[c] = c < dk ? N[c] : 0.f;
    for (int c = tid - MT_C; c < VB * 64; c += ML_THREADS - MT_C) norm_s[c] = c < vn ? a.norm[(size_t)h * dv + v0 + c] : 0.f;
  }
  cp_async_wait<(KB > 1 ? 2 : 1)>();
  fence_proxy_async_smem();
  __syncthreads();
  tmem_fence_after();
  const uint32_t tm = tmem_slot, tm_s = tm, tm_o = tm + MT_C;
  const uint32_t lane_base = (uint32_t)(warp % 4 * 32) << 16;
  const int np = (vn + 15) / 16 * 16;
  const uint32_t idesc_s = mma_idesc(MT_C, MT_C, false, false), idesc_o = mma_idesc(MT_C, np, false, true);
  const uint64_t q_desc = desc_k_major(q_sm, MT_C, 0), k_desc = desc_k_major(k_sm, MT_C, 0);
  const int k_steps = (dk + 15) / 16;
  bool dead = false;  // a wait ran out: wait no more, finish and report
  if (tid == 0) {
#pragma unroll
    for (int k = 0; k < KB * 4; ++k) {
      const uint32_t step = (k / 4) * (MT_BLOCK / 16) + (k % 4) * 2;  // descriptor units of 16 bytes
      if (k < k_steps) mma_ss(tm_s, q_desc + step, k_desc + step, idesc_s, k > 0);
    }
    mma_commit(&bar_s);
  }
  // q . n_in, each half of the threads one half of the channels (while the scores are made)
  float den = 0.f;
  for (int ch = half * KB * 4; ch < (half + 1) * KB * 4; ++ch) {
    float f[8];
    unpack_chunk<bf16>(*reinterpret_cast<const uint4 *>(base + sw128_offset(MT_C, r, ch)), f);
#pragma unroll
    for (int e = 0; e < 8; ++e) den = fmaf(f[e], n_in[ch * 8 + e], den);
  }
  const float win = w_in[r];
  den *= win;
  dead = !mbar_wait(&bar_s, 0);
  __syncwarp();
  tmem_fence_after();
  {
    uint32_t s[2][32];
#pragma unroll
    for (int q = 0; q < 2; ++q) tmem_ld32(s[q], tm_s + lane_base + half * 64 + q * 32);
    tmem_wait_ld();
    tmem_fence_before();  // both halves have read S before either puts P over it
    __syncthreads();
    tmem_fence_after();
    const float2 M = mt[r];
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      uint32_t hi[16], lo[16];
#pragma unroll
      for (int e = 0; e < 32; e += 2) {
        float p[2];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          const int col = half * 64 + q * 32 + e + x;
          const float2 av = as[col];
          const float w = exp2_fast((av.x - M.x) + (av.y - M.y));
          p[x] = col <= r ? __uint_as_float(s[q][e + x]) * (w * a.scale) : 0.f;
          den += p[x];
        }
        split_pair(p[0], p[1], hi[e / 2], lo[e / 2]);
      }
      tmem_st16(tm_s + lane_base + half * 32 + q * 16, hi);
      tmem_st16(tm_s + lane_base + 64 + half * 32 + q * 16, lo);
    }
  }
  exch[half][r] = den;
  tmem_wait_st();
  tmem_fence_before();
  // the incoming state, 64 channels at a time
#pragma unroll
  for (int s = 0; s < KB; ++s) {
    if (s + 1 < KB) cp_async_wait<1>();
    else cp_async_wait<0>();
    fence_proxy_async_smem();
    __syncthreads();
    if (tid == 0) {
      tmem_fence_after();
      const uint32_t buf = buf_sm + (s & 1) * BUF;
#pragma unroll
      for (int part = 0; part < 2; ++part) {
        const uint64_t sd = desc_mn_major(buf + part * VB * SLICE, 64, 0);
#pragma unroll
        for (int k = 0; k < 4; ++k)
          if (s * 4 + k < k_steps)
            mma_ss(tm_o, q_desc + s * (MT_BLOCK / 16) + k * 2, sd + (uint64_t)(k * 128), idesc_o, s + part + k > 0);
      }
      mma_commit(&bar_buf[s & 1]);
    }
    if (s + 2 < KB) {
      if (!dead) dead = !mbar_wait(&bar_buf[s & 1], (s / 2) & 1);
      slice(s + 2);
    }
  }
  constexpr int VBUF = KB & 1;  // free once the slice before the last is done
  if (KB > 1 && !dead) dead = !mbar_wait(&bar_buf[VBUF], ((KB - 2) / 2) & 1);
  load_tile<VB, MT_C>(buf_sm + VBUF * BUF, v_rows, a.ld, cl, vn);
  cp_async_commit();
  if (!dead) dead = !mbar_wait(&bar_buf[(KB - 1) & 1], ((KB - 1) / 2) & 1);
  // the gates take the last slice's buffer
  load_tile<VB, MT_C>(buf_sm + (VBUF ^ 1) * BUF, gate, a.ld, cl, vn);
  cp_async_commit();
  __syncwarp();
  tmem_fence_after();
#pragma unroll 2
  for (int q = half * 16; q < np; q += 64) {  // two groups of 16 columns at a time
    const bool two = q + 32 < np;
    uint32_t o[2][16];
    tmem_ld16(o[0], tm_o + lane_base + q);
    if (two) tmem_ld16(o[1], tm_o + lane_base + q + 32);
    tmem_wait_ld();
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int e = 0; e < 16; ++e) o[x][e] = __float_as_uint(__uint_as_float(o[x][e]) * win);
    tmem_st16(tm_o + lane_base + q, o[0]);
    if (two) tmem_st16(tm_o + lane_base + q + 32, o[1]);
  }
  tmem_wait_st();
  tmem_fence_before();
  cp_async_wait<1>();  // V
  fence_proxy_async_smem();
  __syncthreads();
  if (tid == 0) {
    tmem_fence_after();
    const uint64_t vd = desc_mn_major(buf_sm + VBUF * BUF, MT_C, 0);
#pragma unroll
    for (int k = 0; k < MT_C / 16; ++k) mma_ts(tm_o, tm_s + k * 8, vd + (uint64_t)(k * 128), idesc_o, true);
#pragma unroll
    for (int k = 0; k < MT_C / 16; ++k) mma_ts(tm_o, tm_s + 64 + k * 8, vd + (uint64_t)(k * 128), idesc_o, true);
    mma_commit(&bar_o);
  }
  const float inv = 1.f / (fmaxf(fabsf(exch[0][r] + exch[1][r]), floor_s[r]) + 1e-6f);
  if (!dead) dead = !mbar_wait(&bar_o, 0);
  __syncwarp();
  tmem_fence_after();
  float ss = 0.f;
#pragma unroll 2
  for (int q = half * 16; q < np; q += 64) {
    const bool two = q + 32 < np;
    uint32_t o[2][16];
    tmem_ld16(o[0], tm_o + lane_base + q);
    if (two) tmem_ld16(o[1], tm_o + lane_base + q + 32);
    tmem_wait_ld();
#pragma unroll
    for (int x = 0; x < 2; ++x)
#pragma unroll
      for (int e = 0; e < 16; ++e) {
        const float v = x == 0 || two ? __uint_as_float(o[x][e]) * inv : 0.f;  // (columns past the end are zero)
        ss = fmaf(v, v, ss);
      }
  }
  cp_async_wait<0>();  // the gates
  __syncthreads();     // everybody has read exch
  exch[half][r] = ss;
  __syncthreads();
  float tot = exch[0][r] + exch[1][r];
  if (nvt > 1) {
    cluster.barrier_wait();
    if (half == 0)
      for (int x = 0; x < nvt; ++x) cluster.map_shared_rank(&ssq[0][0], x)[vt * MT_C + r] = tot;
    cluster.sync();
    tot = 0.f;
    for (int x = 0; x < nvt; ++x) tot += ssq[x][r];
  }
  const float rn = inv / sqrtf(tot / (float)dv + a.eps);
  // results go over their gates in shared memory, and out of there row by row
  unsigned char *io = base + 2 * KB * MT_BLOCK + (VBUF ^ 1) * BUF;
#pragma unroll 2
  for (int q = half * 16; q < np; q += 32) {
    uint32_t o[16];
    tmem_ld16(o, tm_o + lane_base + q);
    tmem_wait_ld();
#pragma unroll
    for (int e = 0; e < 16; e += 8) {
      uint4 *p = reinterpret_cast<uint4 *>(io + sw128_offset(MT_C, r, (q + e) / 8));
      float z[8], f[8];
      unpack_chunk<bf16>(*p, z);
#pragma unroll
      for (int x = 0; x < 8; ++x)
        f[x] = __uint_as_float(o[e + x]) * rn * norm_s[q + e + x] * __fdividef(1.f, 1.f + __expf(-z[x]));
      uint4 v;
      v.x = pack_bf16(f[0], f[1]);
      v.y = pack_bf16(f[2], f[3]);
      v.z = pack_bf16(f[4], f[5]);
      v.w = pack_bf16(f[6], f[7]);
      *p = v;
    }
  }
  __syncthreads();
  bf16 *out = static_cast<bf16 *>(a.out) + (((size_t)b * a.n + t0) * a.H + h) * dv + v0;
  for (int i = tid; i < cl * VB * 8; i += ML_THREADS) {
    const int t = i / (VB * 8), ch = i - t * (VB * 8);
    if (ch * 8 < vn)
      *reinterpret_cast<uint4 *>(out + (size_t)t * a.H * dv + ch * 8) = *reinterpret_cast<const uint4 *>(io + sw128_offset(MT_C, t, ch));
  }
  if (dead && tid == 0) atomicAdd(&g_mlstm_timeouts, 1u);
  tmem_fence_before();
  __syncthreads();
  if (warp == 0) tmem_dealloc(tm, COLS);
}

// value blocks of 64 columns per thread block: as many as shared memory and a block's share of TMEM hold
static int out_vb(int dk, int dv) {
  const int kb = ceil_div(dk, 64), want = dv <= 64 ? 1 : (dv <= 128 ? 2 : 4);
  return kb > 2 && want > 2 ? 2 : want;
}

bool mlstm_tc_supported(int dtype, int dk, int dv) {
  return dtype == DJV_DTYPE_BF16 && dk % 8 == 0 && dv % 8 == 0 && dk <= 256 && ceil_div(dv, out_vb(dk, dv) * 64) <= MT_MAX_TILES;
}

int mlstm_tc_gates(const MlstmArgs &a, cudaStream_t st) {
  djv::launch_kernel(mlstm_tc_gates_kernel, dim3(ceil_div(a.nc, MG_WARPS), a.H, a.B), dim3(MG_WARPS * WARP), 0, st, a);
  count_launch();
  return check_launch("mlstm_prefill");
}

int mlstm_tc_chunk_state(const MlstmArgs &a, cudaStream_t st) {
  const int kb = a.dk <= 128 ? 2 : 4, vb = a.dv <= 64 ? 1 : 2, nvt = ceil_div(a.dv, vb * 64);
  const size_t smem = 1024 + (size_t)(2 * kb + vb) * MT_BLOCK;
  const dim3 grid(a.nc * nvt, a.H, a.B);
#define DJV_GO(K_, V_)                                                                                                     \
  if (kb == K_ && vb == V_) {                                                                                              \
    cudaFuncSetAttribute(mlstm_tc_chunk_state_kernel<K_, V_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);     \
    djv::launch_kernel(mlstm_tc_chunk_state_kernel<K_, V_>, grid, dim3(ML_THREADS), smem, st, a, nvt);                     \
  }
  DJV_GO(2, 1)
  DJV_GO(2, 2)
  DJV_GO(4, 1)
  DJV_GO(4, 2)
#undef DJV_GO
  count_launch();
  return check_launch("mlstm_prefill");
}

int mlstm_tc_chunk_out(const MlstmArgs &a, cudaStream_t st) {
  const int kb = ceil_div(a.dk, 64), vb = out_vb(a.dk, a.dv), nvt = ceil_div(a.dv, vb * 64);
  size_t smem = 1024 + (size_t)(2 * kb + 2 * vb) * MT_BLOCK;
  // no more blocks per multiprocessor than TMEM has room for: two, or one with four value blocks
  const size_t least = (vb > 2 ? 120 : 80) * 1024;
  if (smem < least) smem = least;
  DJV_REQUIRE((long long)a.H * a.B <= 65535 && a.nc <= 65535, "mlstm_prefill: too many heads, sequences or chunks");
  const dim3 grid(nvt, a.nc, a.H * a.B);
#define DJV_GO(K_, V_)                                                                                                     \
  if (kb == K_ && vb == V_) {                                                                                              \
    cudaFuncSetAttribute(mlstm_tc_chunk_out_kernel<K_, V_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);       \
    djv::launch_kernel_cluster(mlstm_tc_chunk_out_kernel<K_, V_>, grid, dim3(ML_THREADS), smem, st, dim3(nvt, 1, 1), a);   \
  }
  DJV_GO(1, 1)
  DJV_GO(1, 2)
  DJV_GO(1, 4)
  DJV_GO(2, 1)
  DJV_GO(2, 2)
  DJV_GO(2, 4)
  DJV_GO(3, 1)
  DJV_GO(3, 2)
  DJV_GO(4, 1)
  DJV_GO(4, 2)
#undef DJV_GO
  count_launch();
  return check_launch("mlstm_prefill");
}

}  // namespace djv

extern "C" unsigned djv_mlstm_timeouts(void) {
  unsigned v = 0;
  if (cudaMemcpyFromSymbol(&v, djv::g_mlstm_timeouts, sizeof(v)) != cudaSuccess) {
    cudaGetLastError();
    return 0;
  }
  return v;
}
