// Attention with mixed heads of large prompt portions, on tcgen05 (see gqa_mix.cuh).  Two launches:
//
//   mix_stats_kernel   per head and up to 256 queries of a portion: scores Q K^T in tensor memory, their maximum and sum per
//                      query; leaves log2 of the softmax denominator, [row][head]
//   mix_attn_kernel    one CTA has nq queries of all heads and walks the key tiles they see.  Scores are taken transposed, so
//                      that all heads of a query lie side by side for the thread that owns a key:
//                        S_c [128 keys][nq x group]  = K_c Q_c^T          (kv head c; K tile is the M operand)
//                        p = 2^(s scale - denominator), p'_h = sum_g T[h, g] p_g
//                        O_c [vdim][nq x group]     += V_c^T P'_c         (P' as bf16 through shared memory)
//                      Warp 0 loads K and V tiles of one kv head at a time, warp 1 issues the products, sixteen warps (a key a
//                      lane, four warps share a key's queries; eight for more than 16 heads) turn scores into weights.  Groups of
//                      three heads and more are mixed on mma.sync (f16 operands, f32 sums; the weights are staged where the mixed
//                      ones will stand), smaller ones with packed f32 multiply-adds.  The scores of the next tile are
//                      issued ahead of the values of this one, so the softmax runs beside the value products.
//
// Key tiles are 128 positions (two pages): the tiles of the kept keys, then the window's.  Every wait is bounded.
#include <cuda_fp16.h>
#include <math.h>

#include <algorithm>
#include <type_traits>

#include "act.cuh"
#include "gqa_mix.cuh"
#include "ptx.cuh"
#include "tc.cuh"

namespace rewb {

extern int64_t g_launch_total;

namespace {

constexpr int BOX = 128 * 128;        // 128 rows x 64 bf16 columns
constexpr int TILE = 128;
constexpr float LOG2E = 1.4426950408889634f;
constexpr size_t kSmemMax = 227 * 1024;

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// D(16x8,f32) += A(16x16,f16,row) * B(16x8,f16,col)
__device__ __forceinline__ void mma_f16_16816(float* c, const uint32_t* a, uint32_t b0, uint32_t b1) {
  asm volatile(
      "mma.sync.aligned.m16n8k16.row.col.f32.f16.f16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
      : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
      : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_f16(float lo, float hi) {
  const __half2 v = __floats2half2_rn(lo, hi);
  return *reinterpret_cast<const uint32_t*>(&v);
}
// Two f32 multiply-adds
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
  uint64_t d;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
  return d;
}
__device__ __forceinline__ uint64_t pair2(float x, float y) {
  uint64_t d;
  asm("mov.b64 %0, {%1, %2};" : "=l"(d) : "f"(x), "f"(y));
  return d;
}
__device__ __forceinline__ float2 split2(uint64_t v) {
  float2 d;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(d.x), "=f"(d.y) : "l"(v));
  return d;
}
// N consecutive 32-bit columns of this thread's lane, without the wait
template <int N>
__device__ __forceinline__ void ld_cols(uint32_t taddr, uint32_t* r) {
  if constexpr (N == 2)
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x2.b32 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(taddr) : "memory");
  else if constexpr (N == 4)
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x4.b32 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(taddr) : "memory");
  else if constexpr (N == 8)
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7])
                 : "r"(taddr)
                 : "memory");
  else
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]),
                   "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
                 : "r"(taddr)
                 : "memory");
}

struct PreArgs {
  GqaDims m;
  const GqaTile* tiles;    // up to 256 queries of one portion each
  const float* gate;       // see GqaMixArgs
  int nsplit;
  int64_t split_stride, ld;
  const float* gate_head;
  bf16* out;
  int64_t ldo;
  const int* block_table;
  int max_pages;
  float* lse;              // [row][heads]
  int nb_k, nb_v, stages;
  int nq, nc;              // mix_attn_kernel: queries of a CTA, columns of a kv head
  int* status;
};

// The key tiles that queries at pos_first .. pos_last see.
struct KeyTiles {
  int kept, w0, n;
  __device__ __forceinline__ int at(int i) const { return i < kept ? i : w0 + i - kept; }
};
__device__ __forceinline__ KeyTiles key_tiles(const GqaDims& m, int pos_first, int pos_last) {
  const int lo = m.window > 0 ? max(0, pos_first - m.window + 1) : 0, w0 = lo / TILE;
  const int kept = min((m.keep_first + TILE - 1) / TILE, w0);
  return KeyTiles{kept, w0, kept + pos_last / TILE - w0 + 1};
}
// Whether any of the queries at first .. last sees a key of tile k.
__device__ __forceinline__ bool sees_tile(const GqaDims& m, int k, int first, int last) {
  return k * TILE <= last && (m.window == 0 || k * TILE + TILE - 1 > first - m.window || k * TILE < m.keep_first);
}
// One kv head's tile: two pages, `boxes` boxes each.
__device__ __forceinline__ void load_tile(const PreArgs& a, uint8_t* dst, const CUtensorMap& tm, uint64_t* bar, int lane, int hk, int tile, int boxes) {
  mbar_expect_tx(bar, boxes * BOX);
#pragma unroll
  for (int p = 0; p < 2; ++p) {
    const int page = a.block_table[(int64_t)lane * a.max_pages + min(2 * tile + p, a.max_pages - 1)];
    for (int b = 0; b < boxes; ++b) tma_load_2d(dst + b * BOX + p * 8192, &tm, bar, b * 64, (page * a.m.kv_heads + hk) * 64);
  }
}

// ------------------------------------------------------------------ softmax denominators
// grid (tiles, heads).  Two query tiles share the key tiles; tensor memory holds two score buffers of each.
__global__ void __launch_bounds__(64 + 512, 1) mix_stats_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k,
                                                               const __grid_constant__ PreArgs a) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int nb = a.nb_k, tb = nb * BOX;
  uint8_t* sQ = smem;                                   // two query tiles
  uint8_t* ring = smem + 2 * tb;
  float2* xs = reinterpret_cast<float2*>(ring + a.stages * tb);    // [2][128] of the upper half of the keys
  uint64_t* bars = reinterpret_cast<uint64_t*>(xs + 256);
  uint64_t *k_full = bars, *k_empty = bars + 4, *s_full = bars + 8, *s_free = bars + 12;   // s_*: [query tile][buffer]
  uint64_t* q_full = bars + 16;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 17);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, head = blockIdx.y, hk = head / (a.m.heads / a.m.kv_heads);
  if (threadIdx.x == 0) {
    for (int i = 0; i < 4; ++i) {
      mbar_init(k_full + i, 1);
      mbar_init(k_empty + i, 1);
      mbar_init(s_full + i, 1);
      mbar_init(s_free + i, 8);
    }
    mbar_init(q_full, 1);
    fence_barrier_init();
    pdl_launch_dependents();
  }
  if (warp == 1) tc::alloc(tmem_slot, 512);
  tc::fence_before();
  __syncthreads();
  tc::fence_after();
  const uint32_t tmem = *tmem_slot;
  pdl_wait();
  const GqaTile et = a.tiles[blockIdx.x];
  const KeyTiles kt = key_tiles(a.m, et.pos0, et.pos0 + et.n - 1);
  const int nt = et.n > 128 ? 2 : 1;                    // query tiles
  float m = -INFINITY, l = 0.f;
  if (warp == 0) {
    if (lane == 0) {
      bool ok = true;
      mbar_expect_tx(q_full, nt * tb);
      for (int t = 0; t < nt; ++t)
        for (int b = 0; b < nb; ++b) tma_load_3d(sQ + t * tb + b * BOX, &tm_q, q_full, b * 64, head, et.row0 + t * 128);
      for (int j = 0; j < kt.n && ok; ++j) {
        const int s = j % a.stages;
        if (j >= a.stages) ok = mbar_wait(k_empty + s, (j / a.stages - 1) & 1, a.status);
        if (ok) load_tile(a, ring + s * tb, tm_k, k_full + s, et.lane, hk, kt.at(j), nb);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(TILE >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
      constexpr uint32_t hi = tc::desc_hi(1024);
      const uint32_t q_lo = tc::desc_lo(smem_u32(sQ), 16), k_lo = tc::desc_lo(smem_u32(ring), 16);
      bool ok = mbar_wait(q_full, 0, a.status);
      int it[2] = {0, 0};                               // tiles a query tile has seen so far
      for (int j = 0; j < kt.n && ok; ++j) {
        const int s = j % a.stages;
        ok = mbar_wait(k_full + s, (j / a.stages) & 1, a.status);
        for (int t = 0; t < nt && ok; ++t) {
          const int first = et.pos0 + t * 128;
          if (!sees_tile(a.m, kt.at(j), first, first + min(et.n - t * 128, 128) - 1)) continue;
          const int buf = it[t] & 1, turn = it[t]++ / 2;
          if (turn > 0) ok = mbar_wait(s_free + 2 * t + buf, (turn - 1) & 1, a.status);
          if (!ok) break;
          tc::fence_after();
          for (int b = 0; b < nb; ++b)
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
              const uint32_t off = b * (BOX >> 4) + kk * 2;
              tc::umma_bf16_ss_lh(tmem + t * 256 + buf * 128, q_lo + t * (tb >> 4) + off, k_lo + s * (tb >> 4) + off, hi, idesc, (b > 0 || kk > 0) ? 1u : 0u);
            }
          tc::commit(s_full + 2 * t + buf);
        }
        if (ok) tc::commit(k_empty + s);
      }
    }
  } else {
    const int t = (warp - 2) >> 3, quarter = warp & 3, half = ((warp - 2) >> 2) & 1, row = quarter * 32 + lane;
    if (t < nt) {
      const uint32_t base = tmem + ((uint32_t)(quarter * 32) << 16) + t * 256 + half * 64;
      const int first = et.pos0 + t * 128, last = first + min(et.n - t * 128, 128) - 1, W = a.m.window;
      const int hi = first + row, lo = W > 0 ? hi - W : -1;
      const float sl2 = a.m.scale * LOG2E;
      bool ok = true;
      int it = 0;
      for (int j = 0; j < kt.n; ++j) {
        if (!sees_tile(a.m, kt.at(j), first, last)) continue;
        const int buf = it & 1, turn = it++ / 2, k0 = kt.at(j) * TILE, kh = k0 + half * 64;
        if (ok) ok = mbar_wait(s_full + 2 * t + buf, turn & 1, a.status);
        __syncwarp();
        tc::fence_after();
        uint32_t r0[32], r1[32];
        tc::ld32_issue(base + buf * 128, r0);
        tc::ld32_issue(base + buf * 128 + 32, r1);
        tc::wait_ld();
        tc::fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(s_free + 2 * t + buf);
        if (k0 + TILE - 1 > first || (W > 0 && k0 <= last - W)) {
#pragma unroll
          for (int e = 0; e < 32; ++e) {
            const int ka = kh + e, kb = kh + 32 + e;
            if (ka > hi || (ka <= lo && ka >= a.m.keep_first)) r0[e] = 0xff800000u;            // -inf
            if (kb > hi || (kb <= lo && kb >= a.m.keep_first)) r1[e] = 0xff800000u;
          }
        }
        float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
        for (int e = 0; e < 32; ++e) mx[e & 3] = fmaxf(fmaxf(mx[e & 3], __uint_as_float(r0[e])), __uint_as_float(r1[e]));
        const float mn = fmaxf(m, fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3])) * sl2), use = mn == -INFINITY ? 0.f : mn;   // the host requires a positive scale
        float ls[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int e = 0; e < 32; ++e) ls[e & 3] += ex2(fmaf(__uint_as_float(r0[e]), sl2, -use)) + ex2(fmaf(__uint_as_float(r1[e]), sl2, -use));
        l = l * ex2(m - use) + ((ls[0] + ls[1]) + (ls[2] + ls[3]));
        m = mn;
      }
      if (half) xs[t * 128 + row] = make_float2(m, l);
    }
  }
  tc::fence_before();
  __syncthreads();
  if (warp >= 2) {
    const int t = (warp - 2) >> 3, half = ((warp - 2) >> 2) & 1, row = (warp & 3) * 32 + lane;
    if (!half && t * 128 + row < et.n) {
      const float2 e = xs[t * 128 + row];
      const float M = fmaxf(m, e.x), use = M == -INFINITY ? 0.f : M;
      a.lse[(int64_t)(et.row0 + t * 128 + row) * a.m.heads + head] = use + log2f(l * ex2(m - use) + e.y * ex2(e.x - use));
    }
  }
  if (warp == 1) {
    tc::fence_after();
    tc::dealloc(tmem, 512);
  }
}

// ------------------------------------------------------------------ weights, mixing, values
template <int HP>
struct MixT {
  float2 t[HP * HP / 2];   // by padded head: kv head * G2 + head of its group
};
constexpr int warpgroups(int hp) { return hp <= 16 ? 4 : 2; }   // of the softmax: registers for more heads in fewer threads

// grid (blocks of nq queries).  HP: padded heads at most, G2: heads of a kv head, padded to a power of two.
template <int HP, int G2>
__global__ void __launch_bounds__(64 + 128 * warpgroups(HP), 1) mix_attn_kernel(const __grid_constant__ CUtensorMap tm_q, const __grid_constant__ CUtensorMap tm_k,
                                                               const __grid_constant__ CUtensorMap tm_v, const __grid_constant__ PreArgs a, const __grid_constant__ MixT<HP> T) {
  constexpr int KV = HP / G2;          // kv heads at most
  constexpr int LW = 2 * G2;           // score columns of a pair of queries and a kv head
  constexpr int NW = warpgroups(HP), NTS = 128 * NW;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int G = a.m.kv_heads, group = a.m.heads / G, nc = a.nc, nq = a.nq, nbk = a.nb_k, nbv = a.nb_v;
  const int q_bytes = nc * nbk * 128, st_bytes = max(nbk, nbv) * BOX, p_tiles = (G * nc + 63) / 64;
  uint8_t* sQ = smem;                                   // [kv head][box][nc rows][128 bytes]
  uint8_t* sP = sQ + (G * q_bytes + 1023) / 1024 * 1024;      // [64 columns][128 keys][128 bytes]
  uint8_t* ring = sP + p_tiles * BOX;
  float* sL = reinterpret_cast<float*>(ring + a.stages * st_bytes);   // [nq][HP] minus the denominators
  float2* sT = reinterpret_cast<float2*>(sL + nq * HP);               // [HP][HP] mixing matrix
  uint64_t* bars = reinterpret_cast<uint64_t*>(sT + HP * HP / 2);
  uint64_t *full = bars, *empty = bars + 8, *s_full = bars + 16, *s_free = bars + 17, *p_full = bars + 18, *p_free = bars + 19;
  uint64_t *q_full = bars + 20, *g_full = bars + 21, *o_full = bars + 22;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 23);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < 8; ++i) {
      mbar_init(full + i, 1);
      mbar_init(empty + i, 1);
    }
    mbar_init(s_full, 1);
    mbar_init(s_free, 4 * NW);
    mbar_init(p_full, 4 * NW);
    mbar_init(p_free, 1);
    mbar_init(q_full, 1);
    mbar_init(g_full, 1);
    mbar_init(o_full, 1);
    fence_barrier_init();
    pdl_launch_dependents();
  }
  if (warp == 1) tc::alloc(tmem_slot, 512);
  tc::fence_before();
  __syncthreads();
  tc::fence_after();
  const uint32_t tmem = *tmem_slot;
  const bool bulk = a.gate && a.nsplit == 1;           // gates arrive by bulk copies
  pdl_wait();
  const int per_tile = 256 / nq;
  const GqaTile et = a.tiles[blockIdx.x / per_tile];
  const int skip = (int)(blockIdx.x % per_tile) * nq, n = min(et.n - skip, nq), row0 = et.row0 + skip, pos0 = et.pos0 + skip;   // n may be <= 0 (uniform)
  const KeyTiles kt = n > 0 ? key_tiles(a.m, pos0, pos0 + n - 1) : KeyTiles{0, 0, 0};
  if (warp >= 2 && n > 0) {
    const int idx = threadIdx.x - 64;
    if (a.gate) {   // the gates of the output are on their way to L2 meanwhile
      const int lines = (a.m.heads * a.m.vdim + 31) / 32;
      for (int i = idx; i < n * lines * a.nsplit; i += NTS) {
        const int s = i / (n * lines), r = i / lines % n;
        prefetch_l2(a.gate + s * a.split_stride + (int64_t)(row0 + r) * a.ld + (i % lines) * 32);
      }
    }
    for (int i = idx; i < HP * HP / 2; i += NTS) sT[i] = T.t[i];
    for (int i = idx; i < nq * HP; i += NTS) {
      const int qi = i / HP, g = i % HP, c = g / G2, hh = g % G2;
      // heads and queries that do not exist have a weight of zero
      sL[i] = qi < n && c < G && hh < group ? -a.lse[(int64_t)(row0 + qi) * a.m.heads + c * group + hh] : -INFINITY;
    }
    asm volatile("bar.sync 1, %0;" ::"n"(NTS) : "memory");
  }

  if (warp == 0) {
    if (lane == 0 && n > 0) {
      bool ok = true;
      int cnt = 0;
      // column q * G2 + hh of kv head c: G2 heads from its first one on (those behind its last are never weighed)
      mbar_expect_tx(q_full, G * q_bytes);
      for (int c = 0; c < G; ++c)
        for (int b = 0; b < nbk; ++b) tma_load_3d(sQ + c * q_bytes + b * nc * 128, &tm_q, q_full, b * 64, c * group, row0);
      auto load = [&](bool val, int j) {
        for (int c = 0; c < G && ok; ++c, ++cnt) {
          const int s = cnt % a.stages;
          if (cnt >= a.stages) ok = mbar_wait(empty + s, (cnt / a.stages - 1) & 1, a.status);
          if (ok) load_tile(a, ring + s * st_bytes, val ? tm_v : tm_k, full + s, et.lane, c, kt.at(j), val ? nbv : nbk);
        }
      };
      load(false, 0);
      for (int j = 0; j < kt.n && ok; ++j) {
        if (j + 1 < kt.n) load(false, j + 1);
        load(true, j);
      }
      if (bulk && ok && mbar_wait(o_full, 0, a.status)) {
        const uint32_t bytes = (uint32_t)(a.m.heads * a.m.vdim) * 4;
        mbar_expect_tx(g_full, n * bytes);
        for (int q = 0; q < n; ++q) bulk_load_1d(smem + q * bytes, a.gate + (int64_t)(row0 + q) * a.ld, bytes, g_full);
      }
    }
  } else if (warp == 1) {
    if (lane == 0 && n > 0) {
      const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(nc >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
      const uint32_t idesc_pv = idesc | (1u << 15) | (1u << 16);          // both operands with the contracted index outermost
      constexpr uint32_t hi = tc::desc_hi(1024);
      const uint32_t q_lo = tc::desc_lo(smem_u32(sQ), 16), k_lo = tc::desc_lo(smem_u32(ring), 16);
      const uint32_t v_lo = tc::desc_lo(smem_u32(ring), nbv > 1 ? BOX : 0), p_lo = tc::desc_lo(smem_u32(sP), BOX);
      bool ok = mbar_wait(q_full, 0, a.status);
      int cnt = 0;
      auto scores = [&](int j) {
        if (j > 0) ok = mbar_wait(s_free, (j - 1) & 1, a.status);
        for (int c = 0; c < G && ok; ++c, ++cnt) {
          const int s = cnt % a.stages;
          ok = mbar_wait(full + s, (cnt / a.stages) & 1, a.status);
          if (!ok) break;
          tc::fence_after();
          for (int b = 0; b < nbk; ++b)
#pragma unroll
            for (int kk = 0; kk < 4; ++kk)
              tc::umma_bf16_ss_lh(tmem + c * nc, k_lo + s * (st_bytes >> 4) + b * (BOX >> 4) + kk * 2, q_lo + c * (q_bytes >> 4) + b * (nc * 128 >> 4) + kk * 2, hi, idesc,
                                  (b > 0 || kk > 0) ? 1u : 0u);
          tc::commit(empty + s);
        }
        if (ok) tc::commit(s_full);
      };
      if (ok) scores(0);
      for (int j = 0; j < kt.n && ok; ++j) {
        if (j + 1 < kt.n) scores(j + 1);
        if (ok) ok = mbar_wait(p_full, j & 1, a.status);
        for (int c = 0; c < G && ok; ++c, ++cnt) {
          const int s = cnt % a.stages, col = c * nc;
          ok = mbar_wait(full + s, (cnt / a.stages) & 1, a.status);
          if (!ok) break;
          tc::fence_after();
          const uint32_t pb = p_lo + (col >> 6) * (BOX >> 4) + ((col & 63) * 2 >> 4);
#pragma unroll
          for (int kk = 0; kk < 8; ++kk)
            tc::umma_bf16_ss_lh(tmem + 256 + col, v_lo + s * (st_bytes >> 4) + kk * (2048 >> 4), pb + kk * (2048 >> 4), hi, idesc_pv, (j > 0 || kk > 0) ? 1u : 0u);
          tc::commit(empty + s);
        }
        if (ok) tc::commit(j + 1 < kt.n ? p_free : o_full);
      }
    }
  } else if (n > 0) {
    const int wg = (warp - 2) >> 2, quarter = warp & 3, krow = quarter * 32 + lane, pairs = nq / 2;
    const uint32_t s_addr = tmem + ((uint32_t)(quarter * 32) << 16);
    // the mixing matrix as B operand: heads 8 x + lane / 4 of the output, 16 s + 2 (lane % 4) (+ 8) of the input
    uint32_t tb[HP / 8][HP / 16][2];
    if constexpr (G2 >= 4)
#pragma unroll
      for (int x = 0; x < HP / 8; ++x)
#pragma unroll
        for (int s = 0; s < HP / 16; ++s)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const float2 t = sT[(x * 8 + (lane >> 2)) * (HP / 2) + s * 8 + e * 4 + (lane & 3)];
            tb[x][s][e] = pack_f16(t.x, t.y);
          }
    const uint64_t sl2 = pair2(a.m.scale * LOG2E, a.m.scale * LOG2E);
    const int W = a.m.window;
    bool ok = true;
    for (int j = 0; j < kt.n; ++j) {
      const int k0 = kt.at(j) * TILE, key = k0 + krow;
      const bool edge = k0 + TILE - 1 > pos0 || (W > 0 && k0 <= pos0 + n - 1 - W);
      if (ok) ok = mbar_wait(s_full, j & 1, a.status);
      __syncwarp();
      tc::fence_after();
      // two pairs of queries at a time: their weights are taken to registers first, which frees the scores for the next tile
#pragma unroll 1
      for (int i0 = wg; i0 < pairs; i0 += 2 * NW) {
        // [pair][query][two heads]: f16 for mma.sync, or f32
        std::conditional_t<(G2 >= 4), uint32_t, uint64_t> pw[2][2][HP / 2];
#pragma unroll
        for (int b = 0; b < 2; ++b) {
          const int i = i0 + b * NW;
          if (i >= pairs) break;
          auto& p = pw[b];
          uint32_t r[KV][LW];
#pragma unroll
          for (int c = 0; c < KV; ++c)
            if (c < G) ld_cols<LW>(s_addr + c * nc + i * LW, r[c]);
            else
#pragma unroll
              for (int x = 0; x < LW; ++x) r[c][x] = 0u;     // kv heads that do not exist
          tc::wait_ld();
          // weights, two heads at a time
#pragma unroll
          for (int q = 0; q < 2; ++q) {
            const ulonglong2* L = reinterpret_cast<const ulonglong2*>(sL + (2 * i + q) * HP);
#pragma unroll
            for (int g = 0; g < HP; g += 4) {
              const ulonglong2 e = L[g / 4];
#pragma unroll
              for (int u = 0; u < 2; ++u) {
                const int h0 = g + 2 * u, h1 = h0 + 1;
                const float s0 = __uint_as_float(r[h0 / G2][q * G2 + h0 % G2]), s1 = __uint_as_float(r[h1 / G2][q * G2 + h1 % G2]);
                const float2 x = split2(fma2(pair2(s0, s1), sl2, u ? e.y : e.x));
                if constexpr (G2 >= 4) p[q][h0 / 2] = pack_f16(ex2(x.x), ex2(x.y));
                else p[q][h0 / 2] = pair2(ex2(x.x), ex2(x.y));
              }
            }
            if (edge) {
              const int pos = pos0 + 2 * i + q;
              if (key > pos || (W > 0 && key <= pos - W && key >= a.m.keep_first))
#pragma unroll
                for (int g = 0; g < HP / 2; ++g) p[q][g] = 0;
            }
          }
        }
        if (i0 + 2 * NW >= pairs) {
          tc::fence_before();
          __syncwarp();
          if (lane == 0) mbar_arrive(s_free);
        }
        if (j > 0 && i0 == wg) {
          if (ok) ok = mbar_wait(p_free, (j - 1) & 1, a.status);   // the products of the tile before have read their weights
          __syncwarp();
        }
#pragma unroll
        for (int b = 0; b < 2; ++b) {
          const int i = i0 + b * NW;
          if (i >= pairs) break;
          auto& p = pw[b];
          // 16-byte chunk x of this key and pair of queries: kv head x / (G2 / 4), four heads of it of both queries, or (G2 8) eight of one
          auto chunk = [&](int row, int x) {
            const int col = x / (LW / 8) * nc + i * LW + x % (LW / 8) * 8;
            return sP + (col >> 6) * BOX + swz128((uint32_t)row, (uint32_t)((col & 63) >> 3));
          };
          if constexpr (G2 >= 4) {
            // the weights of both queries pass through the place of the mixed ones: query q, heads 8 x .. in chunk q cq + x
            const int cq = (G * G2 + 7) / 8;
            uint32_t f[2][2][HP / 16][4];    // [query][16 keys][step]
#pragma unroll
            for (int q = 0; q < 2; ++q)
#pragma unroll
              for (int x = 0; x < HP / 8; ++x)
                if (x < cq) *reinterpret_cast<uint4*>(chunk(krow, q * cq + x)) = make_uint4(p[q][4 * x], p[q][4 * x + 1], p[q][4 * x + 2], p[q][4 * x + 3]);
            __syncwarp();
#pragma unroll
            for (int q = 0; q < 2; ++q)
#pragma unroll
              for (int m = 0; m < 2; ++m)
#pragma unroll
                for (int s = 0; s < HP / 16; ++s) {
                  uint32_t(&d)[4] = f[q][m][s];
                  ldmatrix_x4(d[0], d[1], d[2], d[3], smem_u32(chunk(quarter * 32 + m * 16 + (lane & 15), q * cq + min(2 * s + (lane >> 4), cq - 1))));
                  if (2 * s >= cq) d[0] = d[1] = 0u;       // heads that do not exist
                  if (2 * s + 1 >= cq) d[2] = d[3] = 0u;
                }
            __syncwarp();
#pragma unroll
            for (int q = 0; q < 2; ++q)
#pragma unroll
              for (int m = 0; m < 2; ++m)
#pragma unroll
                for (int x = 0; x < HP / 8; ++x) {
                  if (x * 8 / G2 >= G) break;
                  float o[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                  for (int s = 0; s < HP / 16; ++s) mma_f16_16816(o, f[q][m][s], tb[x][s][0], tb[x][s][1]);
                  // rows lane / 4 and + 8, heads 2 (lane % 4) and the next
                  const int h = x * 8 + 2 * (lane & 3), col = h / G2 * nc + (2 * i + q) * G2 + h % G2, r = quarter * 32 + m * 16 + (lane >> 2);
                  if (h / G2 < G) {
                    uint8_t* d = sP + (col >> 6) * BOX + (col & 7) * 2;
                    *reinterpret_cast<uint32_t*>(d + swz128((uint32_t)r, (uint32_t)((col & 63) >> 3))) = pack_bf16(o[0], o[1]);
                    *reinterpret_cast<uint32_t*>(d + swz128((uint32_t)(r + 8), (uint32_t)((col & 63) >> 3))) = pack_bf16(o[2], o[3]);
                  }
                }
            __syncwarp();
          } else {
          const ulonglong2* t = reinterpret_cast<const ulonglong2*>(sT);
#pragma unroll 1
          for (int c = 0; c < G; ++c) {
            float w[LW];     // [query][head of the group]
#pragma unroll
            for (int hh = 0; hh < G2; ++hh) {
              uint64_t w0 = 0ull, w1 = 0ull;     // sums over the even and the odd heads
#pragma unroll
              for (int g = 0; g < HP / 4; ++g) {
                const ulonglong2 e = *t++;
                w0 = fma2(e.x, p[0][2 * g], w0);
                w1 = fma2(e.x, p[1][2 * g], w1);
                w0 = fma2(e.y, p[0][2 * g + 1], w0);
                w1 = fma2(e.y, p[1][2 * g + 1], w1);
              }
              const float2 a0 = split2(w0), a1 = split2(w1);
              w[hh] = a0.x + a0.y;
              w[G2 + hh] = a1.x + a1.y;
            }
            const int col = c * nc + i * LW;
            uint8_t* dst = sP + (col >> 6) * BOX + swz128((uint32_t)krow, (uint32_t)((col & 63) >> 3));
            if constexpr (LW == 2) {
              *reinterpret_cast<uint32_t*>(dst + (col & 7) * 2) = pack_bf16(w[0], w[1]);
            } else if constexpr (LW == 4) {
              *reinterpret_cast<uint2*>(dst + (col & 7) * 2) = make_uint2(pack_bf16(w[0], w[1]), pack_bf16(w[2], w[3]));
            } else {
              *reinterpret_cast<uint4*>(dst) = make_uint4(pack_bf16(w[0], w[1]), pack_bf16(w[2], w[3]), pack_bf16(w[4], w[5]), pack_bf16(w[6], w[7]));
              if constexpr (LW == 16) {
                const int c2 = col + 8;
                *reinterpret_cast<uint4*>(sP + (c2 >> 6) * BOX + swz128((uint32_t)krow, (uint32_t)((c2 & 63) >> 3))) =
                    make_uint4(pack_bf16(w[8], w[9]), pack_bf16(w[10], w[11]), pack_bf16(w[12], w[13]), pack_bf16(w[14], w[15]));
              }
            }
          }
          }
        }
      }
      fence_proxy_async();
      __syncwarp();
      if (lane == 0) mbar_arrive(p_full);
    }
    // ---- output: every product is done, so the shared memory takes the gates and the gated rows, [query][head][value]
    if (ok) ok = mbar_wait(o_full, 0, a.status);
    if (bulk && ok) ok = mbar_wait(g_full, 0, a.status);
    __syncwarp();
    tc::fence_after();
    const int V = a.m.vdim, HV = a.m.heads * V, v = krow;
    const float* const sG = reinterpret_cast<const float*>(smem);
    bf16* const sO = reinterpret_cast<bf16*>(smem + (bulk ? nq * HV * 4 : 0));
    const float* const zg = a.gate + (int64_t)row0 * a.ld + v;      // gates that were not copied
    for (int i = wg; i < pairs && 2 * i < n; i += NW) {
      const bool two = 2 * i + 1 < n;
#pragma unroll 1
      for (int c = 0; c < G; ++c) {
        uint32_t o[LW];
        float z[LW];
        ld_cols<LW>(s_addr + 256 + c * nc + i * LW, o);
        const int at = 2 * i * HV + c * group * V + v;
        auto on = [&](int x) { return x % G2 < group && (x < G2 || two); };   // uniform over the warp
#pragma unroll
        for (int x = 0; x < LW; ++x) z[x] = 0.f;
        if (bulk) {
          if (v < V)
#pragma unroll
            for (int x = 0; x < LW; ++x)
              if (on(x)) z[x] = sG[at + x / G2 * HV + x % G2 * V];
        } else if (a.gate && v < V) {
          for (int s = 0; s < a.nsplit; ++s)
#pragma unroll
            for (int x = 0; x < LW; ++x)
              if (on(x)) z[x] += zg[s * a.split_stride + (2 * i + x / G2) * a.ld + (c * group + x % G2) * V];
        }
        tc::wait_ld();
#pragma unroll
        for (int x = 0; x < LW; ++x) {
          float y = __uint_as_float(o[x]) * a.m.out_scale;
          if (a.gate_head && on(x)) y *= a.gate_head[(int64_t)(row0 + 2 * i + x / G2) * a.m.heads + c * group + x % G2];
          if (a.gate) y = __fdividef(y, 1.0f + ex2(-LOG2E * z[x]));
          if (v < V && on(x)) sO[at + x / G2 * HV + x % G2 * V] = __float2bfloat16_rn(y);
        }
      }
    }
    fence_proxy_async();
    asm volatile("bar.sync 1, %0;" ::"n"(NTS) : "memory");
    if (warp == 2 && ok) {
      for (int q = lane; q < n; q += 32) {
        asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(a.out + (int64_t)(row0 + q) * a.ldo), "r"(smem_u32(sO + q * HV)),
                     "r"((uint32_t)(HV * 2))
                     : "memory");
      }
      asm volatile("cp.async.bulk.commit_group;" ::: "memory");
      asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
    }
  }
  tc::fence_before();
  __syncthreads();
  if (warp == 1) {
    tc::fence_after();
    tc::dealloc(tmem, 512);
  }
}

// How the queries of a CTA and the heads lie side by side.
struct Shape {
  int hp, g2, nq, nc;
};
bool shape_of(const GqaDims& m, Shape* s) {
  const int group = m.heads / m.kv_heads;
  s->g2 = 1;
  while (s->g2 < group) s->g2 *= 2;
  if (s->g2 == 4 && m.kv_heads == 1) s->g2 = 8;   // room to stage the weights
  const int heads = m.kv_heads * s->g2;
  s->hp = heads <= 16 ? 16 : 32;
  if (heads > 32 || s->g2 > 8) return false;
  s->nq = 64 / s->g2;
  while (s->nq * heads > 256 || s->nq > 32) s->nq /= 2;
  s->nc = s->nq * s->g2;
  return s->nc >= 16 && s->nq >= 2;
}
size_t stats_smem(int nb, int stages) { return (size_t)(2 + stages) * nb * BOX + 256 * sizeof(float2) + 256 + 1024; }
size_t attn_smem(const GqaDims& m, const Shape& s, int nbk, int nbv, int stages) {
  return ((size_t)m.kv_heads * s.nc * nbk * 128 + 1023) / 1024 * 1024 + (size_t)((m.kv_heads * s.nc + 63) / 64) * BOX + (size_t)stages * std::max(nbk, nbv) * BOX +
         (size_t)(s.nq + s.hp) * s.hp * 4 + 256 + 1024;
}

}  // namespace

bool gqa_mix_prefill_ok(const GqaDims& m) {
  Shape s;
  return m.dim % 8 == 0 && m.vdim % 8 == 0 && m.dim <= 128 && m.vdim <= 128 && m.scale > 0.f && !m.bias && !m.sink && !m.talk_wide && shape_of(m, &s);
}

int gqa_mix_prefill_launch(Ctx* c, const GqaMixArgs& g, const GqaTile* tiles, int count, const float* talk_host, float* lse) {
  if (count == 0) return REWB200_OK;
  Shape s;
  RB_REQUIRE(gqa_mix_prefill_ok(g.m) && g.dtype == REWB200_BF16 && shape_of(g.m, &s), "attention with mixed heads: sizes without a tcgen05 kernel");
  PreArgs a;
  memset(&a, 0, sizeof(a));
  a.m = g.m;
  a.tiles = tiles;
  a.gate = g.gate;
  a.nsplit = g.nsplit;
  a.split_stride = g.split_stride;
  a.ld = g.ld;
  a.gate_head = g.gate_head;
  a.out = (bf16*)g.out;
  a.ldo = g.ldo;
  a.block_table = g.block_table;
  a.max_pages = g.max_pages;
  a.lse = lse;
  a.nb_k = (g.m.dim + 63) / 64;
  a.nb_v = (g.m.vdim + 63) / 64;
  a.nq = s.nq;
  a.nc = s.nc;
  a.status = g.status;
  CUtensorMap tm_q;
  auto queries = [&](uint32_t box_heads, uint32_t box_rows) {
    return make_tmap_3d_bf16(&tm_q, g.q, (uint64_t)g.m.dim, (uint64_t)g.m.heads, (uint64_t)g.rows, (uint64_t)g.m.dim * 2, (uint64_t)g.ldq * 2, 64, box_heads, box_rows);
  };
  RB_TRY(queries(1, 128));
  a.stages = 4;
  size_t smem = stats_smem(a.nb_k, a.stages);
  RB_CUDA(cudaFuncSetAttribute(mix_stats_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  RB_CUDA(launch_k(mix_stats_kernel, dim3((unsigned)count, (unsigned)g.m.heads), dim3(64 + 512), smem, c->stream, c->use_pdl, tm_q, *g.tm_k, a));
  ++g_launch_total;
  RB_TRY(queries((uint32_t)s.g2, (uint32_t)s.nq));
  a.stages = 8;
  while (a.stages > 2 && attn_smem(g.m, s, a.nb_k, a.nb_v, a.stages) > kSmemMax) --a.stages;
  smem = attn_smem(g.m, s, a.nb_k, a.nb_v, a.stages);
  RB_REQUIRE(smem - (size_t)(s.nq + s.hp) * s.hp * 4 - 1280 >= (size_t)s.nq * g.m.heads * g.m.vdim * 6, "attention with mixed heads: no room for the output rows");
  RB_REQUIRE(smem <= kSmemMax, "attention with mixed heads: shared memory");
  const dim3 grid((unsigned)(count * (256 / s.nq)));
  auto go = [&](auto kernel, auto T, int threads) -> int {
    const int group = g.m.heads / g.m.kv_heads, H = g.m.heads;
    memset(&T, 0, sizeof(T));
    for (int h = 0; h < H; ++h)
      for (int x = 0; x < H; ++x) {
        const int r = h / group * s.g2 + h % group, k = x / group * s.g2 + x % group;
        (k % 2 ? T.t[(r * s.hp + k) / 2].y : T.t[(r * s.hp + k) / 2].x) = talk_host ? talk_host[(int64_t)h * H + x] : h == x ? 1.f : 0.f;
      }
    RB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    RB_CUDA(launch_k(kernel, grid, dim3(threads), smem, c->stream, c->use_pdl, tm_q, *g.tm_k, *g.tm_v, a, T));
    ++g_launch_total;
    return REWB200_OK;
  };
#define RB_MIX1(HP, G2) go(mix_attn_kernel<HP, G2>, MixT<HP>(), 64 + 128 * warpgroups(HP))
#define RB_MIX(HP) (s.g2 == 1 ? RB_MIX1(HP, 1) : s.g2 == 2 ? RB_MIX1(HP, 2) : s.g2 == 4 ? RB_MIX1(HP, 4) : RB_MIX1(HP, 8))
  return s.hp == 16 ? RB_MIX(16) : RB_MIX(32);
#undef RB_MIX
#undef RB_MIX1
}

}  // namespace rewb
