// The chunk kernels of gated linear attention on tensor cores (bf16 projections).
//
// Products whose operand is an fp32 quantity (keys and queries times decays, states, score matrices) take it as two
// bf16 terms, hi + lo, and keep three of the four partial products (two where the other operand is bf16 already): the
// recurrence stays within 2^-16 of fp32. mma.sync tiles rather than the TMEM path: the operands are made in registers
// (decays times keys, states split on the way from global memory), and the 16-row granularity is what the triangular
// score matrix needs.
#include "../../include/dejavu_b200_hybrid.h"
#include "hybrid_gla.cuh"

namespace djv {

constexpr int GC = GLA_MMA_CHUNK;  // tokens per chunk
constexpr int GW = GLA_THREADS / WARP;

__host__ __device__ __forceinline__ int up16(int v) { return (v + 15) & ~15; }

// x, y -> packed bf16 pairs hi and lo with hi + lo = (x, y) to 2^-17
__device__ __forceinline__ void split2(float x, float y, uint32_t &hi, uint32_t &lo) {
  hi = pack_bf16(x, y);
  const float2 r = b2f(hi);
  lo = pack_bf16(x - r.x, y - r.y);
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  mma_m16n8k16_t<bf16>(d, a[0], a[1], a[2], a[3], b0, b1);
}

// rows x cols of bf16 from global (row stride ld) into shared memory, zeros up to pad_rows / pad_cols. 16-byte chunks.
__device__ __forceinline__ void stage_rows(bf16 *dst, int pitch, const bf16 *src, long long ld, int rows, int cols,
                                           int pad_cols) {
  const int chunks = pad_cols / 8, step = GLA_THREADS / chunks;  // (pad_cols <= 256)
  const int r0 = threadIdx.x / chunks, c = threadIdx.x - r0 * chunks;
  if (r0 >= step) return;
  const bool inside = c * 8 < cols;
  const bf16 *s = src + (size_t)r0 * ld + c * 8;
  uint32_t d = smem_addr(dst + r0 * pitch + c * 8);
  for (int r = r0; r < GC; r += step, s += (size_t)step * ld, d += step * pitch * 2) {
    const bool ok = inside && r < rows;
    cp_async16_zfill(d, ok ? s : src, ok ? 16 : 0);
  }
}

// exp, log and sigmoid on the fast units: absolute errors near 2^-23, for quantities that end in bf16 products
__device__ __forceinline__ float log_sigmoid_fast(float z) { return fminf(z, 0.f) - __logf(1.f + __expf(-fabsf(z))); }
__device__ __forceinline__ float silu_fast(float g) { return __fdividef(g, 1.f + __expf(-g)); }

// ---- a chunk's own contribution to the state: U = sum_t (k_t exp(B_C - B_t)) v_t^T, and the sums B_t ----------------
__global__ void __launch_bounds__(GLA_THREADS, 2) gla_mma_chunk_state_kernel(GlaArgs a) {
  extern __shared__ __align__(16) unsigned char sm_raw[];
  pdl_prologue();
  const int tid = threadIdx.x, lane = tid % WARP, warp = tid / WARP;
  const int ci = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const int dk = a.dk, dv = a.dv, dkp = up16(dk), dvp = up16(dv);
  const int kp = dkp + 8, vp = dvp + 8;
  const int t0 = ci * GC, cl = min(GC, a.n - t0);
  bf16 *k_hi = reinterpret_cast<bf16 *>(sm_raw), *k_lo = k_hi + GC * kp, *vs = k_lo + GC * kp;
  float *bs = reinterpret_cast<float *>(vs + GC * vp);  // [GC][dkp]
  float *tot = bs + GC * dkp, *ts = tot + 4 * dkp;      // [4][dkp]; 16 ranks of the decay input at a time: [GC][16]
  const bf16 *rows = static_cast<const bf16 *>(a.proj) + ((size_t)b * a.n + t0) * a.ld;
  const int koff = a.H * dk + h * dk, voff = 2 * a.H * dk + h * dv, toff = 2 * a.H * dk + 2 * a.H * dv;

  stage_rows(k_lo, kp, rows + koff, a.ld, cl, dk, dkp);  // (split in place below)
  stage_rows(vs, vp, rows + voff, a.ld, cl, dv, dvp);
  cp_async_commit();
  // log decays: thread = channel, the rows in steps
  const int cpr = min(dkp, GLA_THREADS), steps = GLA_THREADS / cpr;  // (dk <= 256)
  const int tc = tid % cpr, tr = tid / cpr;
  const float *wr = a.a2 + (size_t)(h * dk + min(tc, dk - 1)) * a.rank;
  for (int r0 = 0; r0 < a.rank; r0 += 16) {
    const int rn = min(16, a.rank - r0);
    __syncthreads();
    for (int i = tid; i < GC * 16; i += GLA_THREADS) {
      const int t = i / 16, r = i % 16;
      ts[i] = (t < cl && r < rn) ? to_f(rows[(size_t)t * a.ld + toff + r0 + r]) : 0.f;
    }
    __syncthreads();
    if (tc < dk && tr < steps) {
      float w[16];
#pragma unroll
      for (int r = 0; r < 16; ++r) w[r] = r < rn ? __ldg(wr + r0 + r) : 0.f;
      const float bias = a.a2_bias[h * dk + tc];
      const bool last = r0 + 16 >= a.rank;
      for (int t = tr; t < GC; t += steps) {
        float z = r0 == 0 ? bias : bs[t * dkp + tc];
#pragma unroll
        for (int r = 0; r < 16; r += 4) {
          const float4 x = *reinterpret_cast<const float4 *>(ts + t * 16 + r);
          z = fmaf(x.x, w[r], z);
          z = fmaf(x.y, w[r + 1], z);
          z = fmaf(x.z, w[r + 2], z);
          z = fmaf(x.w, w[r + 3], z);
        }
        // tokens past the end change nothing: their decay is 1
        bs[t * dkp + tc] = last ? (t < cl ? log_sigmoid_fast(z) * a.inv_tau : 0.f) : z;
      }
    }
  }
  __syncthreads();
  // sums along the chunk: `parts` threads per channel, each over its own stretch first
  const int parts = steps >= 4 ? 4 : (steps >= 2 ? 2 : 1), len = GC / parts;
  if (tc < dk && tr < parts) {
    float run = 0.f;
#pragma unroll 16
    for (int t = tr * len; t < tr * len + len; ++t) {
      run += bs[t * dkp + tc];
      bs[t * dkp + tc] = run;
    }
    tot[tr * dkp + tc] = run;
  }
  __syncthreads();
  if (tc < dk && tr < parts) {
    float before = 0.f;
    for (int x = 0; x < tr; ++x) before += tot[x * dkp + tc];
    if (tr > 0) {
#pragma unroll 16
      for (int t = tr * len; t < tr * len + len; ++t) bs[t * dkp + tc] += before;
    }
    if (tr == parts - 1) a.decay[(((size_t)b * a.H + h) * a.nc + ci) * dk + tc] = before + tot[tr * dkp + tc];
  }
  cp_async_wait<0>();
  __syncthreads();
  const int kc = dkp / 2, kstep = GLA_THREADS / kc;  // pairs of channels, rows at a time
  const int kt0 = tid / kc, c2 = (tid - kt0 * kc) * 2;
  if (kt0 < kstep) {
    const bool inside = c2 < dk;  // dk is even
    const float2 e = inside ? *reinterpret_cast<const float2 *>(bs + (GC - 1) * dkp + c2) : make_float2(0.f, 0.f);
    float *cum = a.cum + (((size_t)b * a.n + t0 + kt0) * a.H + h) * dk + c2;
#pragma unroll 4
    for (int t = kt0; t < GC; t += kstep, cum += (size_t)kstep * a.H * dk) {
      float x = 0.f, y = 0.f;
      if (t < cl && inside) {
        const float2 s = *reinterpret_cast<const float2 *>(bs + t * dkp + c2);
        const float2 k = b2f(*reinterpret_cast<const uint32_t *>(k_lo + t * kp + c2));
        x = k.x * __expf(e.x - s.x);
        y = k.y * __expf(e.y - s.y);
        *reinterpret_cast<float2 *>(cum) = s;
      }
      uint32_t hi, lo;
      split2(x, y, hi, lo);
      *reinterpret_cast<uint32_t *>(k_hi + t * kp + c2) = hi;
      *reinterpret_cast<uint32_t *>(k_lo + t * kp + c2) = lo;
    }
  }
  __syncthreads();
  // U (channels x values): a warp takes 16 channels and walks the value columns 16 at a time
  float *U = a.contrib + (((size_t)b * a.H + h) * a.nc + ci) * (size_t)dk * dv;
  const int g = lane / 4, t4 = lane % 4, lm = lane % 8, lq = lane / 8;
  for (int c0 = warp * 16; c0 < dkp; c0 += GW * 16) {
    uint32_t ah[GC / 16][4], al[GC / 16][4];
#pragma unroll
    for (int s = 0; s < GC / 16; ++s) {
      // A (channel, token) from rows of tokens: transposed load; matrices (c 0-7, t 0-7), (c 8-15, t 0-7), (c, t 8-15)
      const int off = (s * 16 + (lq / 2) * 8 + lm) * kp + c0 + (lq % 2) * 8;
      ldmatrix_x4_trans(ah[s], smem_addr(k_hi + off));
      ldmatrix_x4_trans(al[s], smem_addr(k_lo + off));
    }
    for (int j0 = 0; j0 < dvp; j0 += 16) {
      float acc[2][4] = {};
#pragma unroll
      for (int s = 0; s < GC / 16; ++s) {
        uint32_t bv[4];  // (t 0-7, j 0-7), (t 8-15, j 0-7), (t 0-7, j 8-15), (t 8-15, j 8-15)
        ldmatrix_x4_trans(bv, smem_addr(vs + (s * 16 + (lq % 2) * 8 + lm) * vp + j0 + (lq / 2) * 8));
        mma_bf16(acc[0], ah[s], bv[0], bv[1]);
        mma_bf16(acc[1], ah[s], bv[2], bv[3]);
        mma_bf16(acc[0], al[s], bv[0], bv[1]);
        mma_bf16(acc[1], al[s], bv[2], bv[3]);
      }
#pragma unroll
      for (int x = 0; x < 2; ++x) {
        const int j = j0 + x * 8 + t4 * 2;
        if (j < dv) {  // dv is even
          if (c0 + g < dk) *reinterpret_cast<float2 *>(U + (size_t)(c0 + g) * dv + j) = make_float2(acc[x][0], acc[x][1]);
          if (c0 + g + 8 < dk)
            *reinterpret_cast<float2 *>(U + (size_t)(c0 + g + 8) * dv + j) = make_float2(acc[x][2], acc[x][3]);
        }
      }
    }
  }
}

// ---- a chunk's outputs -----------------------------------------------------------------------------------------------
// scores of 16 query rows (block I) against 8 keys from key j0 on, relative to the sum `ref` before the block:
// q_t exp(B_t - ref) . k_s exp(ref - B_s); the second exponent is <= 0 for keys before the block
template <int NT>  // n-tiles of 8 value columns per warp
__global__ void __launch_bounds__(GLA_THREADS, 2) gla_mma_chunk_out_kernel(GlaArgs a) {
  extern __shared__ __align__(16) unsigned char sm_raw[];
  __shared__ float ssq[GW][GC];
  pdl_prologue();
  const int tid = threadIdx.x, lane = tid % WARP, warp = tid / WARP;
  const int ci = blockIdx.x, h = blockIdx.y, b = blockIdx.z;
  const int dk = a.dk, dv = a.dv, dkp = up16(dk), dvp = up16(dv);
  const int kp = dkp + 8, vp = dvp + 8, bp = dkp + 4, ap = GC + 8;
  const int t0 = ci * GC, cl = min(GC, a.n - t0);
  bf16 *qs = reinterpret_cast<bf16 *>(sm_raw), *ks = qs + GC * kp, *vs = ks + GC * kp;
  float *bs = reinterpret_cast<float *>(vs + GC * vp);            // [GC][bp]
  bf16 *a_hi = reinterpret_cast<bf16 *>(bs), *a_lo = a_hi + GC * ap;  // over bs, once the sums are used up
  const bf16 *rows = static_cast<const bf16 *>(a.proj) + ((size_t)b * a.n + t0) * a.ld;
  const int qoff = h * dk, koff = a.H * dk + h * dk, voff = 2 * a.H * dk + h * dv, goff = voff + a.H * dv;

  // the incoming state is needed last: have it in L2 by then
  const float *S = a.contrib + (((size_t)b * a.H + h) * a.nc + ci) * (size_t)dk * dv;
  for (int i = tid * 32; i < dk * dv; i += GLA_THREADS * 32) prefetch_l2(S + i);
  const int gate_lines = (dv + 63) / 64;  // and the gates
  for (int i = tid; i < cl * gate_lines; i += GLA_THREADS)
    prefetch_l2(rows + (size_t)(i / gate_lines) * a.ld + goff + i % gate_lines * 64);
  stage_rows(qs, kp, rows + qoff, a.ld, cl, dk, dkp);
  stage_rows(ks, kp, rows + koff, a.ld, cl, dk, dkp);
  stage_rows(vs, vp, rows + voff, a.ld, cl, dv, dvp);
  {
    const float *cum = a.cum + (((size_t)b * a.n + t0) * a.H + h) * dk;
    const int per = dkp / 4, step = GLA_THREADS / per;  // dk % 8 == 0
    const int r0 = tid / per, c = (tid - r0 * per) * 4;
    if (r0 < step) {
#pragma unroll 4
      for (int t = r0; t < GC; t += step) {
        // (rows past the end repeat the last sum; columns past the end are zero)
        const bool ok = c < dk;
        cp_async16_zfill(smem_addr(bs + t * bp + c), ok ? cum + (size_t)min(t, cl - 1) * a.H * dk + c : cum, ok ? 16 : 0);
      }
    }
  }
  cp_async_commit();
  cp_async_wait<0>();
  __syncthreads();

  // scores: two warps per block of 16 rows, key tiles of 8 alternate between them
  const int g = lane / 4, t4 = lane % 4, lm = lane % 8, lq = lane / 8;
  const int I = warp / 2, r0 = I * 16;
  constexpr int MAXT = GC / 16;  // key tiles per warp
  float sc[MAXT][4];
#pragma unroll
  for (int x = 0; x < MAXT; ++x)
#pragma unroll
    for (int e = 0; e < 4; ++e) sc[x][e] = 0.f;
  // keys inside the block: their factor exp(ref - B_s) is above 1; it must stay far from overflow
  bool mild = true;
  for (int c = lane; c < dk; c += WARP)
    mild = mild && (I == 0 ? 0.f : bs[(r0 - 1) * bp + c]) - bs[(r0 + 15) * bp + c] < 60.f;
  mild = __all_sync(0xffffffffu, mild);
  for (int k0 = 0; k0 < dkp; k0 += 16) {
    const int ca = k0 + t4 * 2, cb = ca + 8;
    float2 ra = make_float2(0.f, 0.f), rb = ra;  // sums before the block
    if (I > 0) {
      ra = *reinterpret_cast<const float2 *>(bs + (r0 - 1) * bp + ca);
      rb = *reinterpret_cast<const float2 *>(bs + (r0 - 1) * bp + cb);
    }
    uint32_t qh[4], ql[4];
    {
      auto query = [&](int row, int c, const float2 &r, uint32_t &hi, uint32_t &lo) {
        const float2 q = b2f(*reinterpret_cast<const uint32_t *>(qs + row * kp + c));
        const float2 s = *reinterpret_cast<const float2 *>(bs + row * bp + c);
        split2(q.x * a.scale * __expf(s.x - r.x), q.y * a.scale * __expf(s.y - r.y), hi, lo);
      };
      query(r0 + g, ca, ra, qh[0], ql[0]);
      query(r0 + g + 8, ca, ra, qh[1], ql[1]);
      query(r0 + g, cb, rb, qh[2], ql[2]);
      query(r0 + g + 8, cb, rb, qh[3], ql[3]);
    }
#pragma unroll
    for (int x = 0; x < MAXT; ++x) {
      const int j0 = (2 * x + warp % 2) * 8;
      if (j0 < r0 + (mild ? 16 : 0)) {
        uint32_t kh[2], kl[2];
        auto key = [&](int c, const float2 &r, uint32_t &hi, uint32_t &lo) {
          const float2 k = b2f(*reinterpret_cast<const uint32_t *>(ks + (j0 + g) * kp + c));
          const float2 s = *reinterpret_cast<const float2 *>(bs + (j0 + g) * bp + c);
          split2(k.x * __expf(r.x - s.x), k.y * __expf(r.y - s.y), hi, lo);
        };
        key(ca, ra, kh[0], kl[0]);
        key(cb, rb, kh[1], kl[1]);
        mma_bf16(sc[x], qh, kh[0], kh[1]);
        mma_bf16(sc[x], ql, kh[0], kh[1]);
        mma_bf16(sc[x], qh, kl[0], kl[1]);
      }
    }
  }
  if (!mild) {
    // decays too strong for a common reference inside the block: every pair by itself (the tile j0 is x = I here)
    const int j0 = r0 + (warp % 2) * 8;
    float d[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int t = r0 + g + (e / 2) * 8, s = j0 + t4 * 2 + e % 2;
      if (s <= t)
        for (int c = 0; c < dk; ++c)
          d[e] = fmaf(to_f(qs[t * kp + c]) * a.scale * to_f(ks[s * kp + c]), __expf(bs[t * bp + c] - bs[s * bp + c]), d[e]);
    }
#pragma unroll
    for (int x = 0; x < MAXT; ++x)
      if (x == I) {
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[x][e] = d[e];
      }
  }
  __syncthreads();
  // queries for the incoming state: q exp(B_t), split, over q and k
  const int kc = dkp / 2, kstep = GLA_THREADS / kc;
  const int kt0 = tid / kc, c2 = (tid - kt0 * kc) * 2;
  if (kt0 < kstep) {
#pragma unroll 4
    for (int t = kt0; t < GC; t += kstep) {
      const float2 q = b2f(*reinterpret_cast<const uint32_t *>(qs + t * kp + c2));
      const float2 s = *reinterpret_cast<const float2 *>(bs + t * bp + c2);
      uint32_t hi, lo;
      split2(q.x * a.scale * __expf(s.x), q.y * a.scale * __expf(s.y), hi, lo);
      *reinterpret_cast<uint32_t *>(qs + t * kp + c2) = hi;
      *reinterpret_cast<uint32_t *>(ks + t * kp + c2) = lo;
    }
  }
  __syncthreads();
#pragma unroll
  for (int x = 0; x < MAXT; ++x) {
    const int s = (2 * x + warp % 2) * 8 + t4 * 2;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = r0 + g + e * 8;
      uint32_t hi, lo;
      split2(s <= t ? sc[x][2 * e] : 0.f, s + 1 <= t ? sc[x][2 * e + 1] : 0.f, hi, lo);
      *reinterpret_cast<uint32_t *>(a_hi + t * ap + s) = hi;
      *reinterpret_cast<uint32_t *>(a_lo + t * ap + s) = lo;
    }
  }
  __syncthreads();

  // outputs: a warp takes NT * 8 value columns of all 64 rows
  const int n0 = warp * NT * 8;
  float acc[GC / 16][NT][4];
#pragma unroll
  for (int m = 0; m < GC / 16; ++m)
#pragma unroll
    for (int x = 0; x < NT; ++x)
#pragma unroll
      for (int e = 0; e < 4; ++e) acc[m][x][e] = 0.f;
  const int lrow = (lq % 2) * 8 + lm, lcol = (lq / 2) * 8;  // ldmatrix rows of an A operand
  for (int k0 = 0; k0 < dkp; k0 += 16) {
    uint32_t sh[NT][2], sl[NT][2];
#pragma unroll
    for (int x = 0; x < NT; ++x) {
      const int j = n0 + x * 8 + g;
      float v[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int c = k0 + t4 * 2 + (e / 2) * 8 + e % 2;
        v[e] = (j < dv && c < dk) ? __ldg(S + (size_t)c * dv + j) : 0.f;
      }
      split2(v[0], v[1], sh[x][0], sl[x][0]);
      split2(v[2], v[3], sh[x][1], sl[x][1]);
    }
#pragma unroll
    for (int m = 0; m < GC / 16; ++m) {
      uint32_t qh[4], ql[4];
      ldmatrix_x4(qh, smem_addr(qs + (m * 16 + lrow) * kp + k0 + lcol));
      ldmatrix_x4(ql, smem_addr(ks + (m * 16 + lrow) * kp + k0 + lcol));
#pragma unroll
      for (int x = 0; x < NT; ++x) {
        mma_bf16(acc[m][x], qh, sh[x][0], sh[x][1]);
        mma_bf16(acc[m][x], ql, sh[x][0], sh[x][1]);
        mma_bf16(acc[m][x], qh, sl[x][0], sl[x][1]);
      }
    }
  }
#pragma unroll
  for (int s0 = 0; s0 < GC; s0 += 16) {
    uint32_t bv[NT][2];
#pragma unroll
    for (int x = 0; x < NT; ++x) {
      uint32_t r[4];  // (only the first two matrices are used: the addresses of lanes 16..31 repeat them)
      const int col = min(n0 + x * 8, dvp - 8);
      ldmatrix_x4_trans(r, smem_addr(vs + (s0 + (lq % 2) * 8 + lm) * vp + col));
      bv[x][0] = r[0];
      bv[x][1] = r[1];
    }
#pragma unroll
    for (int m = s0 / 16; m < GC / 16; ++m) {
      uint32_t ph[4], pl[4];
      ldmatrix_x4(ph, smem_addr(a_hi + (m * 16 + lrow) * ap + s0 + lcol));
      ldmatrix_x4(pl, smem_addr(a_lo + (m * 16 + lrow) * ap + s0 + lcol));
#pragma unroll
      for (int x = 0; x < NT; ++x) {
        mma_bf16(acc[m][x], ph, bv[x][0], bv[x][1]);
        mma_bf16(acc[m][x], pl, bv[x][0], bv[x][1]);
      }
    }
  }
  // norm over the head's values, gate (whose loads are in flight while the sums meet)
  uint32_t gates[GC / 16][2][NT];
#pragma unroll
  for (int m = 0; m < GC / 16; ++m)
#pragma unroll
    for (int e = 0; e < 2; ++e)
#pragma unroll
      for (int x = 0; x < NT; ++x) {
        const int t = m * 16 + g + e * 8, j = n0 + x * 8 + t4 * 2;
        gates[m][e][x] = (t < cl && j < dv) ? *reinterpret_cast<const uint32_t *>(rows + (size_t)t * a.ld + goff + j) : 0;
      }
#pragma unroll
  for (int m = 0; m < GC / 16; ++m)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      float s = 0.f;
#pragma unroll
      for (int x = 0; x < NT; ++x) {
        const int j = n0 + x * 8 + t4 * 2;
        if (j < dv) s += acc[m][x][2 * e] * acc[m][x][2 * e] + acc[m][x][2 * e + 1] * acc[m][x][2 * e + 1];
      }
      s += __shfl_xor_sync(0xffffffffu, s, 1);
      s += __shfl_xor_sync(0xffffffffu, s, 2);
      if (t4 == 0) ssq[warp][m * 16 + g + e * 8] = s;
    }
  __syncthreads();
#pragma unroll
  for (int m = 0; m < GC / 16; ++m)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int t = m * 16 + g + e * 8;
      if (t >= cl) continue;
      float tot = 0.f;
#pragma unroll
      for (int w = 0; w < GW; ++w) tot += ssq[w][t];
      const float rn = 1.f / sqrtf(tot / (float)dv + a.eps);
      bf16 *out = static_cast<bf16 *>(a.out) + (((size_t)b * a.n + t0 + t) * a.H + h) * dv;
#pragma unroll
      for (int x = 0; x < NT; ++x) {
        const int j = n0 + x * 8 + t4 * 2;
        if (j < dv) {
          const float2 gt = b2f(gates[m][e][x]);
          const float2 w = *reinterpret_cast<const float2 *>(a.norm + j);
          *reinterpret_cast<uint32_t *>(out + j) =
              pack_bf16(acc[m][x][2 * e] * rn * w.x * silu_fast(gt.x), acc[m][x][2 * e + 1] * rn * w.y * silu_fast(gt.y));
        }
      }
    }
}

static size_t mma_state_smem(int dk, int dv) {
  const int dkp = up16(dk), dvp = up16(dv);
  return (size_t)GC * ((2 * (dkp + 8) + dvp + 8) * 2 + dkp * 4) + 4 * dkp * 4 + GC * 16 * 4;
}
static size_t mma_out_smem(int dk, int dv) {
  const int dkp = up16(dk), dvp = up16(dv);
  size_t over = (size_t)GC * (dkp + 4) * 4;
  const size_t scores = (size_t)2 * GC * (GC + 8) * 2;
  if (over < scores) over = scores;
  return (size_t)GC * (2 * (dkp + 8) + dvp + 8) * 2 + over;
}

bool gla_mma_supported(int dtype, int dk, int dv) {
  return dtype == DJV_DTYPE_BF16 && dk % 8 == 0 && dv % 8 == 0 && dk <= 256 && dv <= 256 &&
         mma_state_smem(dk, dv) <= 220 * 1024 && mma_out_smem(dk, dv) <= 220 * 1024;
}

int gla_mma_chunk_state(const GlaArgs &a, cudaStream_t st) {
  const size_t smem = mma_state_smem(a.dk, a.dv);
  cudaFuncSetAttribute(gla_mma_chunk_state_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  djv::launch_kernel(gla_mma_chunk_state_kernel, dim3(a.nc, a.H, a.B), dim3(GLA_THREADS), smem, st, a);
  count_launch();
  return check_launch("gla_prefill");
}

int gla_mma_chunk_out(const GlaArgs &a, cudaStream_t st) {
  const size_t smem = mma_out_smem(a.dk, a.dv);
  const dim3 grid(a.nc, a.H, a.B);
#define DJV_GO(NT_)                                                                                              \
  {                                                                                                              \
    cudaFuncSetAttribute(gla_mma_chunk_out_kernel<NT_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
    djv::launch_kernel(gla_mma_chunk_out_kernel<NT_>, grid, dim3(GLA_THREADS), smem, st, a);                     \
  }
  const int nt = ceil_div(a.dv, 64);
  if (nt == 1) DJV_GO(1)
  else if (nt == 2) DJV_GO(2)
  else if (nt == 3) DJV_GO(3)
  else DJV_GO(4)
#undef DJV_GO
  count_launch();
  return check_launch("gla_prefill");
}

}  // namespace djv
