// Sliding-window attention of a prompt portion on the 5th-generation tensor cores (bf16).
//
// A block takes 128 queries of one head and walks the key tiles of 128 that their windows touch:
//   S (TMEM, 128 x 128 fp32) = Q K^T;  softmax in registers, two threads per query row (64 keys each), no shuffles;
//   P goes back to TMEM over S as two bf16 terms, p = hi + lo, so that the weights keep their fp32 value to 2^-17;
//   O (TMEM, 128 x dv fp32) += P_hi V + P_lo V.
// O is only rescaled when a row's maximum grows by more than 2^8 (the final division by the sum makes up for the rest).
// Keys come from the ring (tokens before the portion) or from the projection's output (the portion's own), or, where the
// caller has put earlier tokens before the portion's, from rows on both sides; the last dimensions of a key may come from
// rows that all heads share. They are fetched row by row, with 16-byte asynchronous copies into the swizzled operand
// layout. Two blocks share a multiprocessor: one computes its softmax while the other's products run. V of a tile loads
// behind its scores, K of the next one behind the values' products.
#include "../../include/dejavu_b200_hybrid.h"
#include "hybrid_attention.cuh"
#include "tcgen05.cuh"

#include <type_traits>

namespace djv {

constexpr int WP_THREADS = 256;
constexpr int WP_TILE = 128;  // queries per block, keys per tile

__device__ unsigned g_window_timeouts;  // bounded waits that ran out (never, in a healthy run)

__device__ __forceinline__ float exp2_approx(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// pairs of floats: one instruction for two
__device__ __forceinline__ uint64_t pack2(float lo, float hi) {
  uint64_t v;
  asm("mov.b64 %0, {%1, %2};" : "=l"(v) : "f"(lo), "f"(hi));
  return v;
}
__device__ __forceinline__ void unpack2(uint64_t v, float &lo, float &hi) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t add2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("add.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}
__device__ __forceinline__ uint64_t sub2(uint64_t a, uint64_t b) {
  uint64_t d;
  asm("sub.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
  return d;
}

template <int KB, int VB>  // 64-element blocks of a query/key row and of a value row
__global__ void __launch_bounds__(WP_THREADS, VB > 2 ? 1 : 2) window_prefill_kernel(WindowArgs a) {
  extern __shared__ unsigned char smem_raw[];
  __shared__ __align__(8) uint64_t bar_s, bar_o;
  __shared__ uint32_t tmem_slot;
  __shared__ float exch[2][WP_TILE];  // maxima, and in the end sums, of the two halves of a row
  constexpr uint32_t COLS = VB > 2 ? 512 : 256;
  constexpr uint32_t KT = KB * WP_TILE * 128;
  const int tid = threadIdx.x, warp = tid / WARP;
  const int half = tid / WP_TILE, r = tid % WP_TILE;  // keys of a tile, query row; warps w and w + 4 share TMEM lanes
  // the first queries of a sequence have short windows: their blocks come last and fill the tail of the grid
  const int h = blockIdx.x, b = blockIdx.z, g = h / (a.H / a.G);
  const int t0 = (int)(gridDim.y - 1 - blockIdx.y) * WP_TILE;
  unsigned char *base = reinterpret_cast<unsigned char *>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
  // with three blocks per key, values go over their keys: two thread blocks fit a multiprocessor that way, and each loads
  // while the other computes
  constexpr bool OVER = KB == 3 && VB <= 2;
  const uint32_t q_sm = smem_u32(base), k_sm = q_sm + KT, v_sm = OVER ? k_sm : k_sm + KT;
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("griddepcontrol.wait;" ::: "memory");

  if (tid == 0) {
    mbar_init(&bar_s, 1);
    mbar_init(&bar_o, 1);
    mbar_fence_init();
  }
  __syncwarp();
  if (warp == 0) tmem_alloc(&tmem_slot, COLS);

  const size_t first = (size_t)b * (a.past + a.n) + a.past;  // row of the portion's first token among the keys
  const int own = a.dk - a.rot, rot = a.rot;  // key dimensions of the head itself, and those all heads share
  const bf16 *q_rows = static_cast<const bf16 *>(a.q) + (size_t)b * a.n * a.ldq + (size_t)h * a.dk;
  const bf16 *k_new = static_cast<const bf16 *>(a.k) + first * a.ldk + (size_t)g * own;
  const bf16 *v_new = static_cast<const bf16 *>(a.v) + first * a.ldv + (size_t)g * a.dv;
  const bf16 *t_new = rot ? static_cast<const bf16 *>(a.tail) + first * a.ldt : k_new;
  const bool ring = a.k_ring != nullptr;  // where the tokens before the portion are: rings, or the rows before the portion's
  const bf16 *kr = ring ? static_cast<const bf16 *>(a.k_ring) + ((size_t)b * a.G + g) * a.cap * a.dk : k_new;
  const bf16 *vr = ring ? static_cast<const bf16 *>(a.v_ring) + ((size_t)b * a.G + g) * a.cap * a.dv : v_new;
  const long long p0 = a.pos[b];
  const int last = min(t0 + WP_TILE, a.n) - 1;
  // everything below is relative to the portion: key j of the portion is token j, the ring holds j < 0
  long long reach = p0 < (long long)a.window - 1 ? p0 : (long long)a.window - 1;  // earlier tokens the portion can see
  if (!ring && reach > a.past) reach = a.past;
  int lo = t0 - (a.window - 1);
  if (lo < -(int)reach) lo = -(int)reach;
  const int tiles = (last - lo) / WP_TILE + 1;
  const int ring_slot0 = (int)((p0 - reach) % a.cap);  // slot of token -reach

  // One tile of keys or values. The chunk a thread copies is the same in every row, so a tile of the portion's own
  // tokens (or of rows before them) is a pointer that advances by a fixed number of rows. Three blocks of 64 elements go
  // one by one, so that a row's chunks are a power of two.
  auto load = [&](uint32_t dst, int j0, const bf16 *ring_rows, int dim, const bf16 *fresh, long long ld, int head_dim,
                  auto blocks) {
    constexpr int NB = decltype(blocks)::value, PASSES = NB == 3 ? 3 : 1;
    constexpr int PER_ROW = NB / PASSES * 8, STEP = WP_THREADS / PER_ROW, ROUNDS = WP_TILE / STEP;
    const int r0 = tid / PER_ROW;
#pragma unroll
    for (int ps = 0; ps < PASSES; ++ps) {
      const int ch = ps * 8 + (tid & (PER_ROW - 1));
      const bool inside = ch * 8 < dim, shared = ch * 8 >= head_dim;
      const bf16 *col = shared ? t_new + (ch * 8 - head_dim) : fresh + ch * 8;
      const long long step1 = shared ? a.ldt : ld;
      if ((!ring || j0 >= 0) && j0 + WP_TILE - 1 <= last) {
        const bf16 *src = inside ? col + (long long)(j0 + r0) * step1 : fresh;  // (not read outside)
        const long long step = (long long)STEP * step1;
#pragma unroll
        for (int it = 0; it < ROUNDS; ++it) {
          cp_async16_zfill(dst + sw128_offset(WP_TILE, r0 + it * STEP, ch), src, inside ? 16 : 0);
          if (inside) src += step;
        }
      } else {
        for (int x = r0; x < WP_TILE; x += STEP) {
          const int j = j0 + x;
          const bf16 *src = fresh;
          const bool ok = inside && j <= last;
          if (ok) {
            if (!ring || j >= 0) {
              src = col + (long long)j * step1;
            } else {
              int slot = ring_slot0 + (j + (int)reach);
              if (slot >= a.cap) slot -= a.cap;
              src = ring_rows + (size_t)slot * dim + ch * 8;
            }
          }
          cp_async16_zfill(dst + sw128_offset(WP_TILE, x, ch), src, ok ? 16 : 0);
        }
      }
    }
    cp_async_commit();
  };
  const std::integral_constant<int, KB> kb;
  const std::integral_constant<int, VB> vb;
  {  // queries
    for (int i = tid; i < WP_TILE * KB * 8; i += WP_THREADS) {
      const int x = i / (KB * 8), ch = i - x * (KB * 8);
      const bool ok = ch * 8 < a.dk && t0 + x <= last;
      cp_async16_zfill(q_sm + sw128_offset(WP_TILE, x, ch), ok ? q_rows + (size_t)(t0 + x) * a.ldq + ch * 8 : q_rows,
                       ok ? 16 : 0);
    }
  }
  load(k_sm, lo, kr, a.dk, k_new, a.ldk, own, kb);

  const float sink = a.sink ? a.sink[h] * 1.4426950408889634f : 0.f;
  const float c = a.scale * 1.4426950408889634f;  // scores in units of log 2
  float m = -1e30f, l = 0.f;
  const int row = t0 + r;
  const uint32_t idesc_s = mma_idesc(WP_TILE, WP_TILE, false, false);
  const int dvp = (a.dv + 15) / 16 * 16;
  const uint32_t idesc_o = mma_idesc(WP_TILE, dvp, false, true);
  const int k_steps = (a.dk + 15) / 16;
  const uint64_t q_desc = desc_k_major(q_sm, WP_TILE, 0), k_desc = desc_k_major(k_sm, WP_TILE, 0);
  const uint64_t v_desc = desc_mn_major(v_sm, WP_TILE, 0);
  bool dead = false;  // a wait ran out: wait no more, finish and report
  __syncthreads();
  tmem_fence_after();
  const uint32_t tm = tmem_slot;
  const uint32_t tm_s = tm, tm_o = tm + WP_TILE;
  const uint32_t lane_base = (uint32_t)(warp % 4 * 32) << 16;

  for (int i = 0; i < tiles; ++i) {
    const int j0 = lo + i * WP_TILE;
    if (i > 0) {  // the last tile's values: P (over S), V and O are free
      if (!dead) dead = !mbar_wait(&bar_o, (i - 1) & 1);
      __syncwarp();  // (TMEM accesses are whole-warp instructions)
      tmem_fence_after();
      if (OVER) load(k_sm, j0, kr, a.dk, k_new, a.ldk, own, kb);
    }
    cp_async_wait<0>();
    fence_proxy_async_smem();
    __syncthreads();
    if (tid == 0) {
      tmem_fence_after();
#pragma unroll
      for (int k = 0; k < KB * 4; ++k) {
        const uint32_t step = (k / 4) * (WP_TILE * 128 / 16) + (k % 4) * 2;  // descriptor units of 16 bytes
        if (k < k_steps) mma_ss(tm_s, q_desc + step, k_desc + step, idesc_s, k > 0);
      }
      mma_commit(&bar_s);
    }
    if (!OVER) load(v_sm, j0, vr, a.dv, v_new, a.ldv, a.dv, vb);
    if (!dead) dead = !mbar_wait(&bar_s, i & 1);
    if (OVER) load(v_sm, j0, vr, a.dv, v_new, a.ldv, a.dv, vb);
    __syncwarp();
    tmem_fence_after();
    __syncwarp();
    uint32_t s[2][32];
#pragma unroll
    for (int q = 0; q < 2; ++q) tmem_ld32(s[q], tm_s + lane_base + half * 64 + q * 32);
    tmem_wait_ld();
    // keys outside this row's window: those after it and those more than window - 1 before it
    const bool edge = j0 + WP_TILE - 1 > t0 || j0 < t0 + WP_TILE - a.window;
    if (edge) {
      const int hi_c = row - j0 - half * 64, lo_c = hi_c - a.window + 1;  // columns lo_c .. hi_c are seen
#pragma unroll
      for (int q = 0; q < 2; ++q)
#pragma unroll
        for (int e = 0; e < 32; ++e)
          if (q * 32 + e > hi_c || q * 32 + e < lo_c) s[q][e] = 0xff800000u;  // -inf
    }
    // (a negative scale turns the maximum round; masked entries stay at -inf below)
    float mx = -INFINITY;
    if (c >= 0.f) {
      float mm[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};  // independent chains
#pragma unroll
      for (int q = 0; q < 2; ++q)
#pragma unroll
        for (int e = 0; e < 32; ++e) mm[e % 4] = fmaxf(mm[e % 4], __uint_as_float(s[q][e]));
      mx = fmaxf(fmaxf(mm[0], mm[1]), fmaxf(mm[2], mm[3]));
    } else {
#pragma unroll
      for (int q = 0; q < 2; ++q)
#pragma unroll
        for (int e = 0; e < 32; ++e)
          if (s[q][e] != 0xff800000u) {
            mx = fmaxf(mx, -__uint_as_float(s[q][e]));
            s[q][e] ^= 0x80000000u;
          }
    }
    exch[half][r] = mx;
    tmem_fence_before();  // both halves have read S before either puts P over it
    __syncthreads();
    tmem_fence_after();
    mx = fmaxf(mx, exch[half ^ 1][r]);
    const float ca = fabsf(c);
    mx *= ca;
    if (a.sink && i == 0) mx = fmaxf(mx, sink);
    const bool grow = mx > m + 8.f;
    if (i == 0) {
      m = fmaxf(mx, m);
      l = a.sink && half == 0 ? exp2_approx(sink - m) : 0.f;
    } else if (__any_sync(0xffffffffu, grow)) {
      const float corr = grow ? exp2_approx(m - mx) : 1.f;
      if (grow) m = mx;
      l *= corr;
      for (int q = half * 16; q < dvp; q += 32) {
        uint32_t o[16];
        tmem_ld16(o, tm_o + lane_base + q);
        tmem_wait_ld();
#pragma unroll
        for (int e = 0; e < 16; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * corr);
        tmem_st16(tm_o + lane_base + q, o);
      }
    }
    const float nm = -m;
    const uint64_t ca2 = pack2(ca, ca), nm2 = pack2(nm, nm);
    uint64_t l2[2] = {0, 0};
#pragma unroll
    for (int q = 0; q < 2; ++q) {
      uint32_t hi[16], lw[16];
#pragma unroll
      for (int e = 0; e < 16; ++e) {
        float x, y;
        unpack2(fma2(pack2(__uint_as_float(s[q][2 * e]), __uint_as_float(s[q][2 * e + 1])), ca2, nm2), x, y);
        x = exp2_approx(x);
        y = exp2_approx(y);
        const uint64_t p = pack2(x, y);
        l2[e % 2] = add2(l2[e % 2], p);
        // hi: the upper halves; the rest, which a float holds exactly, is rounded to bf16
        hi[e] = __byte_perm(__float_as_uint(x), __float_as_uint(y), 0x7632);
        const uint64_t top = pack2(__uint_as_float(__float_as_uint(x) & 0xffff0000u),
                                   __uint_as_float(__float_as_uint(y) & 0xffff0000u));
        float rx, ry;
        unpack2(sub2(p, top), rx, ry);
        lw[e] = pack_bf16(rx, ry);
      }
      tmem_st16(tm_s + lane_base + half * 32 + q * 16, hi);
      tmem_st16(tm_s + lane_base + 64 + half * 32 + q * 16, lw);
    }
    {
      float x, y;
      unpack2(add2(l2[0], l2[1]), x, y);
      l += x + y;
    }
    tmem_wait_st();
    tmem_fence_before();
    cp_async_wait<0>();  // V
    fence_proxy_async_smem();
    __syncthreads();
    if (tid == 0) {
      tmem_fence_after();
#pragma unroll
      for (int k = 0; k < WP_TILE / 16; ++k)
        mma_ts(tm_o, tm_s + k * 8, v_desc + (uint64_t)(k * 128), idesc_o, i > 0 || k > 0);
#pragma unroll
      for (int k = 0; k < WP_TILE / 16; ++k)
        mma_ts(tm_o, tm_s + 64 + k * 8, v_desc + (uint64_t)(k * 128), idesc_o, true);
      mma_commit(&bar_o);
    }
    if (!OVER && i + 1 < tiles) load(k_sm, j0 + WP_TILE, kr, a.dk, k_new, a.ldk, own, kb);  // behind the values' products
  }
  if (!dead) dead = !mbar_wait(&bar_o, (tiles - 1) & 1);
  __syncwarp();
  tmem_fence_after();
  __syncthreads();
  exch[half][r] = l;
  __syncthreads();
  const float inv = 1.f / (l + exch[half ^ 1][r]);
  bf16 *out = static_cast<bf16 *>(a.out) + (((size_t)b * a.n + row) * a.H + h) * a.dv;
  const bf16 *gate = a.gate ? static_cast<const bf16 *>(a.gate) + ((size_t)b * a.n + row) * a.ldg + (size_t)h * a.dv : nullptr;
  for (int q = half * 16; q < dvp; q += 32) {
    uint32_t o[16];
    tmem_ld16(o, tm_o + lane_base + q);
    tmem_wait_ld();
    if (row <= last) {
#pragma unroll
      for (int e = 0; e < 16; e += 8) {
        if (q + e < a.dv) {  // dv % 8 == 0
          float f[8];
#pragma unroll
          for (int x = 0; x < 8; ++x) f[x] = __uint_as_float(o[e + x]) * inv;
          if (gate) {
            float z[8];
            unpack_chunk<bf16>(*reinterpret_cast<const uint4 *>(gate + q + e), z);
#pragma unroll
            for (int x = 0; x < 8; ++x) f[x] *= sigmoid_f(z[x]);
          }
          uint4 v;
          v.x = pack_bf16(f[0], f[1]);
          v.y = pack_bf16(f[2], f[3]);
          v.z = pack_bf16(f[4], f[5]);
          v.w = pack_bf16(f[6], f[7]);
          *reinterpret_cast<uint4 *>(out + q + e) = v;
        }
      }
    }
    __syncwarp();
  }
  if (dead && tid == 0) atomicAdd(&g_window_timeouts, 1u);
  tmem_fence_before();
  __syncthreads();
  if (warp == 0) tmem_dealloc(tm, COLS);
}

template <int KB, int VB>
static int launch_window_prefill(const WindowArgs &a, cudaStream_t st) {
  size_t smem = 1024 + (size_t)(2 * KB + (KB == 3 && VB <= 2 ? 0 : VB)) * WP_TILE * 128;
  // as many blocks per multiprocessor as TMEM has room for: two, or one with wide values
  const size_t least = (VB > 2 ? 120 : 80) * 1024;
  if (smem < least) smem = least;
  cudaFuncSetAttribute(window_prefill_kernel<KB, VB>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
  djv::launch_kernel(window_prefill_kernel<KB, VB>, dim3(a.H, ceil_div(a.n, WP_TILE), a.B), dim3(WP_THREADS), smem, st,
                     a);
  count_launch();
  return check_launch("window_attn");
}

bool window_prefill_supported(const WindowArgs &a) {
  if (!(aligned16(a.k_ring) && aligned16(a.v_ring))) return false;
  if (a.rot && !(a.rot % 8 == 0 && a.ldt % 8 == 0 && aligned16(a.tail))) return false;
  if (a.gate && !(a.ldg % 8 == 0 && aligned16(a.gate))) return false;
  return a.dk % 8 == 0 && a.dv % 8 == 0 && a.dk <= 256 && a.dv <= 256 && a.ldq % 8 == 0 && a.ldk % 8 == 0 &&
         a.ldv % 8 == 0 && aligned16(a.q) && aligned16(a.k) && aligned16(a.v) && aligned16(a.out);
}

int window_prefill(const WindowArgs &a, cudaStream_t st) {
  const int kb = a.dk <= 64 ? 1 : (a.dk <= 128 ? 2 : (a.dk <= 192 ? 3 : 4)), vb = a.dv <= 64 ? 1 : (a.dv <= 128 ? 2 : 4);
#define DJV_WP(K_, V_) \
  if (kb == K_ && vb == V_) return launch_window_prefill<K_, V_>(a, st)
  DJV_WP(1, 1);
  DJV_WP(1, 2);
  DJV_WP(1, 4);
  DJV_WP(2, 1);
  DJV_WP(2, 2);
  DJV_WP(2, 4);
  DJV_WP(3, 1);
  DJV_WP(3, 2);
  DJV_WP(3, 4);
  DJV_WP(4, 1);
  DJV_WP(4, 2);
  return launch_window_prefill<4, 4>(a, st);
#undef DJV_WP
}

}  // namespace djv

extern "C" unsigned djv_window_timeouts(void) {
  unsigned v = 0;
  if (cudaMemcpyFromSymbol(&v, djv::g_window_timeouts, sizeof(v)) != cudaSuccess) {
    cudaGetLastError();
    return 0;
  }
  return v;
}
