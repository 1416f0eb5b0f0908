// Attention of large prompt portions on tcgen05, shared by the mixers that have such a kernel.  A policy P says where
// queries, keys and values come from and what the softmax adds.
//
// A CTA owns one head of up to QT x 128 queries of one portion (QT 2 where shared memory allows it, else 1); both query
// tiles share every 128-key K / V tile.  Warp roles:
//   warp 0        TMA: K tiles and V tiles
//   warp 1        one thread issues S_t = Q_t K^T and O_t += P_t V; while the softmax warps of one query tile work, the
//                 tensor core runs the other tile's products
//   warps 2 ..    eight softmax warps per query tile: thread = query row, two warps share a row's keys.  Scores, biases,
//                 maxima and sums are f32; P goes back to tensor memory as bf16.
// Tensor memory: S_t (P overwrites it) 128 columns each, O_t 64 x value boxes columns each.  Every wait is bounded.
// A query sees the keys of its window only: key tiles outside a query tile's windows are skipped, tiles across an edge
// are masked.
//
// P has
//   kBias                      the scores get an f32 bias by distance
//   sink(head)                 score of the softmax denominator's term without a value, -inf for none
//   tile(i, skip)              tile i without its first `skip` queries: row0, n (may be <= 0), pos0 and what P itself needs
//   k_base(tile)               position of the first key the tile's key tiles count from
//   window()                   keys a query sees, itself included; 0: all
//   q_chunk(tile, qi, head, box, col)   eight score features of a query (16 bytes), zero where there are none
//   load_k / load_v(dst, tm_a, tm_b, bar, tile, head, j, k_base, cf)   issue the TMA loads of key tile j
//   bias_table(head, table), n_bias()      (kBias) fill the table of biases by distance (see bias_slots)
//   and the fields heads, vdim, scale, gate, out, ldo, status.
#pragma once
#include <math.h>

#include "common.cuh"
#include "ptx.cuh"
#include "tc.cuh"

namespace rewb {

extern int64_t g_launch_total;

namespace flash {

constexpr int BOX_BYTES = 128 * 128;   // 128 rows x 64 bf16 columns
constexpr int XCH_FLOATS = 3 * 2 * 128;   // per query tile: two buffers of half-row maxima, half-row sums
constexpr float LOG2E = 1.4426950408889634f;
// A table of biases by distance covers the distances a masked or near tile can have: from -BIAS_PAD (keys after the query,
// -inf) to n_bias - 1 + BIAS_PAD.
constexpr int BIAS_PAD = 254;
constexpr int bias_slots(int n_bias) { return n_bias + 2 * BIAS_PAD; }

struct Cfg {
  int nb_k, nb_v;   // 64-column boxes of score features and of values
  int v_stages;
};

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void pair_barrier(int id) { asm volatile("bar.sync %0, 64;" ::"r"(id) : "memory"); }

// The softmax of one query tile (see attention.cu for the exchange between the two warps of a lane quarter).  Key tiles
// j_lo .. j_hi - 1, tile j = keys k_base + 128 j ..; first / last: positions of the tile's first and last query.
template <class P>
__device__ __forceinline__ void softmax_rows(const P& a, const Cfg& cf, const float* tab, uint32_t s_addr, uint32_t o_addr, float* xmax, float* xsum,
                                             uint64_t* s_full, uint64_t* p_full, uint64_t* o_done, int j_lo, int j_hi, int k_base, int row0,
                                             int n, int first, int quarter, int half, int lane, int pair_bar, int head) {
  const int row = quarter * 32 + lane;
  const int hi = first + row;                                        // last visible key
  const int W = a.window();
  const int lo = W > 0 ? hi - W : -1;                                // the key before the first visible one
  const int last = first + min(n, 128) - 1;
  const float sl2 = a.scale * LOG2E;
  float m, l, far = 0.f;
  if constexpr (P::kBias) far = tab[BIAS_PAD + a.n_bias() - 1];
  m = a.sink(head) * LOG2E;            // the sink: one more term of the denominator, -inf without one
  l = half == 0 && m != -INFINITY ? 1.f : 0.f;
  bool ok = true;
  for (int j = j_lo; j < j_hi; ++j) {
    const int it = j - j_lo;
    if (ok) ok = mbar_wait(s_full, it & 1, a.status);
    __syncwarp();
    tc::fence_after();
    const int kt = k_base + j * 128, k0 = kt + half * 64;
    const bool edge = kt + 127 > first - (P::kBias ? a.n_bias() - 1 : 0) || (W > 0 && kt <= last - W);
    uint32_t r0[32], r1[32];
    tc::ld32_issue(s_addr + half * 64, r0);
    tc::ld32_issue(s_addr + half * 64 + 32, r1);
    tc::wait_ld();
    float sl = sl2, add = far;             // scores in base 2: r * sl + add
    if (P::kBias && edge) {
      const float* tp = tab + BIAS_PAD + hi - k0;
#pragma unroll
      for (int e = 0; e < 32; ++e) {
        r0[e] = __float_as_uint(fmaf(__uint_as_float(r0[e]), sl2, tp[-e]));
        r1[e] = __float_as_uint(fmaf(__uint_as_float(r1[e]), sl2, tp[-32 - e]));
      }
      sl = 1.f;
      add = 0.f;
    } else if (edge) {
#pragma unroll
      for (int e = 0; e < 32; ++e) {
        if (k0 + e > hi || k0 + e <= lo) r0[e] = 0xff800000u;            // -inf
        if (k0 + 32 + e > hi || k0 + 32 + e <= lo) r1[e] = 0xff800000u;
      }
    }
    float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
    for (int e = 0; e < 32; e += 4)
#pragma unroll
      for (int u = 0; u < 4; ++u) mx4[u] = fmaxf(fmaxf(mx4[u], __uint_as_float(r0[e + u])), __uint_as_float(r1[e + u]));
    float mraw = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
    float* xm = xmax + (it & 1) * 256;
    xm[half * 128 + row] = mraw;
    pair_barrier(pair_bar);   // both warps hold their scores in registers now; P may overwrite them
    mraw = fmaxf(mraw, xm[(half ^ 1) * 128 + row]);
    // the maximum of the raw scores is that of the scaled ones: the host requires a positive scale
    const float mx = fmaxf(m, P::kBias ? fmaf(mraw, sl, add) : mraw * sl2);
    const float m_use = mx == -INFINITY ? 0.f : mx;
    const float alpha = ex2(m - m_use), shift = P::kBias ? add - m_use : -m_use;
    float ls[4] = {0.f, 0.f, 0.f, 0.f};
    uint32_t pk[32];
#pragma unroll
    for (int cc = 0; cc < 2; ++cc) {
      const uint32_t* rr = cc ? r1 : r0;
#pragma unroll
      for (int e = 0; e < 32; e += 2) {
        const float p0 = ex2(fmaf(__uint_as_float(rr[e]), P::kBias ? sl : sl2, shift));
        const float p1 = ex2(fmaf(__uint_as_float(rr[e + 1]), P::kBias ? sl : sl2, shift));
        ls[(e >> 1) & 3] += p0 + p1;
        pk[cc * 16 + (e >> 1)] = pack_bf16(p0, p1);
      }
    }
    tc::st32(s_addr + half * 32, pk);
    l = l * alpha + ((ls[0] + ls[1]) + (ls[2] + ls[3]));
    m = mx;
    // S of this tile was announced after P V of the one before it, so O is complete up to there
    if (it > 0 && __any_sync(0xffffffffu, alpha != 1.0f)) {
#pragma unroll 1
      for (int c = 0; c < cf.nb_v; ++c) {
        const uint32_t at = o_addr + half * 32 * cf.nb_v + c * 32;
        tc::ld32_issue(at, r0);
        tc::wait_ld();
#pragma unroll
        for (int e = 0; e < 32; ++e) r0[e] = __float_as_uint(__uint_as_float(r0[e]) * alpha);
        tc::st32_issue(at, r0);
        tc::wait_st();
      }
    }
    tc::fence_before();
    __syncwarp();
    if (lane == 0) mbar_arrive(p_full);
  }
  xsum[half * 128 + row] = l;
  pair_barrier(pair_bar);
  l += xsum[(half ^ 1) * 128 + row];
  const int tiles = j_hi - j_lo;
  if (tiles > 0 && ok) ok = mbar_wait(o_done, (tiles - 1) & 1, a.status);
  __syncwarp();
  tc::fence_after();
  if (tiles <= 0) return;
  const bool store = row < n && ok;
  const int64_t grow = row0 + min(row, n - 1);
  const float gt = a.gate ? a.gate[grow * a.heads + head] : 1.0f;
  const float inv = l > 0.f ? gt / l : 0.f;
  bf16* op = a.out + grow * a.ldo + (int64_t)head * a.vdim;
  uint32_t r[32];
#pragma unroll 1
  for (int c = 0; c < cf.nb_v; ++c) {
    const int col = half * 32 * cf.nb_v + c * 32;
    tc::ld32(o_addr + col, r);
    if (!store) continue;
#pragma unroll
    for (int e = 0; e < 32; e += 8) {
      if (col + e >= a.vdim) continue;   // vdim is a multiple of 8
      uint4 v;
      v.x = pack_bf16(__uint_as_float(r[e]) * inv, __uint_as_float(r[e + 1]) * inv);
      v.y = pack_bf16(__uint_as_float(r[e + 2]) * inv, __uint_as_float(r[e + 3]) * inv);
      v.z = pack_bf16(__uint_as_float(r[e + 4]) * inv, __uint_as_float(r[e + 5]) * inv);
      v.w = pack_bf16(__uint_as_float(r[e + 6]) * inv, __uint_as_float(r[e + 7]) * inv);
      *reinterpret_cast<uint4*>(op + col + e) = v;
    }
  }
}

template <int QT, class P>
__global__ void __launch_bounds__(64 + QT * 256, 1) flash_tc_kernel(const __grid_constant__ CUtensorMap tm_a, const __grid_constant__ CUtensorMap tm_b,
                                                           const __grid_constant__ P a, Cfg cf) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int nb = cf.nb_k;
  const int q_bytes = nb * BOX_BYTES, k_bytes = nb * BOX_BYTES, v_bytes = cf.nb_v * BOX_BYTES;
  uint8_t* sQ = smem;
  uint8_t* sK = sQ + QT * q_bytes;
  uint8_t* sV = sK + k_bytes;
  float* xch = reinterpret_cast<float*>(sV + cf.v_stages * v_bytes);
  uint64_t* bars = reinterpret_cast<uint64_t*>(xch + QT * XCH_FLOATS);
  uint64_t *k_full = bars, *k_empty = bars + 1, *v_full = bars + 2, *v_empty = bars + 4, *s_full = bars + 6, *p_full = bars + 8,
           *o_done = bars + 10;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 12);
  float* tab = reinterpret_cast<float*>(bars + 14);   // kBias: biases by distance
  constexpr uint32_t TM_COLS = QT * 256;

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.y;
  if (threadIdx.x == 0) {
    mbar_init(k_full, 1);
    mbar_init(k_empty, 1);
    for (int i = 0; i < 2; ++i) {
      mbar_init(v_full + i, 1);
      mbar_init(v_empty + i, 1);
      mbar_init(s_full + i, 1);
      mbar_init(p_full + i, 8);
      mbar_init(o_done + i, 1);
    }
    fence_barrier_init();
    pdl_launch_dependents();
  }
  if (warp == 1) tc::alloc(tmem_slot, TM_COLS);
  tc::fence_before();
  __syncthreads();
  tc::fence_after();
  const uint32_t tmem_base = *tmem_slot;
  pdl_wait();

  // QT == 1: two CTAs per listed tile, 128 queries each
  const auto et = a.tile(QT == 2 ? blockIdx.x : blockIdx.x >> 1, QT == 2 ? 0 : (int)(blockIdx.x & 1) * 128);
  const int row0 = et.row0, n = et.n, pos0 = et.pos0;   // n may be <= 0 (uniform over the CTA)
  const int W = a.window();
  const int k_base = a.k_base(et);
  int jlo[2] = {0, 0}, jhi[2] = {0, 0};
#pragma unroll
  for (int t = 0; t < QT; ++t) {
    const int first = pos0 + t * 128, nt = min(n - t * 128, 128);
    if (nt <= 0) continue;
    jlo[t] = W > 0 ? max(0, first - W + 1 - k_base) >> 7 : 0;
    jhi[t] = ((first + nt - 1 - k_base) >> 7) + 1;
  }
  const int j_end = max(jhi[0], jhi[1]);

  if (warp >= 2 && n > 0) {
    // queries: one row per two threads of a tile, in the layout a 128-byte-swizzled TMA would leave
    const int idx = threadIdx.x - 64, r = idx & 127, part = (idx >> 7) & 1, t = idx >> 8;
    const int qi = t * 128 + r;
    for (int ch = part; ch < nb * 8; ch += 2) {
      const int box = ch >> 3;
      const uint4 v = qi < n ? a.q_chunk(et, qi, head, box, (ch & 7) * 8) : make_uint4(0, 0, 0, 0);
      *reinterpret_cast<uint4*>(sQ + t * q_bytes + box * BOX_BYTES + swz128((uint32_t)r, (uint32_t)(ch & 7))) = v;
    }
    if constexpr (P::kBias) a.bias_table(head, tab, (int)threadIdx.x - 64, QT * 256);
    fence_proxy_async();
  }
  __syncthreads();

  if (warp == 0) {
    if (lane == 0 && n > 0) {
      tma_prefetch_desc(&tm_a);
      tma_prefetch_desc(&tm_b);
      bool ok = true;
      for (int j = 0; j < j_end && ok; ++j) {
        if (j > 0) ok = mbar_wait(k_empty, (j - 1) & 1, a.status);
        if (!ok) break;
        mbar_expect_tx(k_full, k_bytes);
        a.load_k(sK, tm_a, tm_b, k_full, et, head, j, k_base, cf);
        const int st = j % cf.v_stages;
        if (j >= cf.v_stages) ok = mbar_wait(v_empty + st, (j / cf.v_stages - 1) & 1, a.status);
        if (!ok) break;
        mbar_expect_tx(v_full + st, v_bytes);
        a.load_v(sV + st * v_bytes, tm_a, tm_b, v_full + st, et, head, j, k_base, cf);
      }
    }
  } else if (warp == 1) {
    if (lane == 0 && n > 0) {
      const uint32_t idesc_qk = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(128 >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);
      const uint32_t idesc_pv = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(cf.nb_v * 8) << 17) | ((uint32_t)(128 >> 4) << 24);
      constexpr uint32_t hi = tc::desc_hi(1024);
      const uint32_t q_lo = tc::desc_lo(smem_u32(sQ), 16), k_lo = tc::desc_lo(smem_u32(sK), 16), v_lo = tc::desc_lo(smem_u32(sV), BOX_BYTES);
      auto active = [&](int t, int j) { return j >= jlo[t] && j < jhi[t]; };
      auto issue_qk = [&](int t) {
        const uint32_t qa = q_lo + t * (q_bytes >> 4);
        for (int b = 0; b < nb; ++b)
#pragma unroll
          for (int kk = 0; kk < 4; ++kk) {
            const uint32_t off = b * (BOX_BYTES >> 4) + kk * 2;
            tc::umma_bf16_ss_lh(tmem_base + t * 128, qa + off, k_lo + off, hi, idesc_qk, (b > 0 || kk > 0) ? 1u : 0u);
          }
        tc::commit(s_full + t);
      };
      bool ok = mbar_wait(k_full, 0, a.status);
      if (ok) {
        tc::fence_after();
#pragma unroll
        for (int t = 0; t < QT; ++t)
          if (active(t, 0)) issue_qk(t);
        tc::commit(k_empty);
      }
      for (int j = 0; j < j_end && ok; ++j) {
        const int st = j % cf.v_stages;
        bool v_ready = false, k_ready = false;
#pragma unroll
        for (int t = 0; t < QT; ++t) {
          if (!ok) break;
          if (active(t, j)) {
            ok = mbar_wait(p_full + t, (j - jlo[t]) & 1, a.status);
            if (ok && !v_ready) ok = v_ready = mbar_wait(v_full + st, (j / cf.v_stages) & 1, a.status);
            if (!ok) break;
            tc::fence_after();
            const uint32_t va = v_lo + st * (v_bytes >> 4);
            const uint32_t acc0 = j > jlo[t] ? 1u : 0u;
#pragma unroll
            for (int kk = 0; kk < 8; ++kk)
              tc::umma_bf16_ta_lh(tmem_base + QT * 128 + t * 128, tmem_base + t * 128 + kk * 8, va + kk * (2048 >> 4), hi, idesc_pv,
                                  kk > 0 ? 1u : acc0);
            tc::commit(o_done + t);
          }
          if (active(t, j + 1)) {
            if (!k_ready) ok = k_ready = mbar_wait(k_full, (j + 1) & 1, a.status);
            if (!ok) break;
            tc::fence_after();
            issue_qk(t);
          }
        }
        if (!ok) break;
        // the query tiles' key ranges overlap or touch, so some tile has waited for these loads already; if none had,
        // the buffers must not be released before they have landed
        if (!v_ready) ok = mbar_wait(v_full + st, (j / cf.v_stages) & 1, a.status);
        if (ok && j + 1 < j_end && !k_ready) ok = mbar_wait(k_full, (j + 1) & 1, a.status);
        if (!ok) break;
        tc::commit(v_empty + st);
        if (j + 1 < j_end) tc::commit(k_empty);
      }
    }
  } else {
    const int t = (warp - 2) >> 3;
    const int quarter = warp & 3, half = ((warp - 2) >> 2) & 1;
    const uint32_t lane_addr = tmem_base + ((uint32_t)(quarter * 32) << 16);
    float* xmax = xch + t * XCH_FLOATS;
    softmax_rows<P>(a, cf, tab, lane_addr + t * 128, lane_addr + QT * 128 + t * 128, xmax, xmax + 2 * 2 * 128, s_full + t, p_full + t, o_done + t,
                 t == 0 ? jlo[0] : jlo[1], t == 0 ? jhi[0] : jhi[1], k_base, row0 + t * 128, n - t * 128, pos0 + t * 128, quarter, half, lane,
                 1 + t * 4 + quarter, head);
  }
  tc::fence_before();
  __syncthreads();
  if (warp == 1) {
    tc::fence_after();
    tc::dealloc(tmem_base, TM_COLS);
  }
}

constexpr size_t kSmemMax = 227 * 1024;

inline size_t smem_bytes(int nb_k, int nb_v, int qt, int v_stages, size_t extra) {
  return (size_t)(qt * nb_k + nb_k + v_stages * nb_v) * BOX_BYTES + (size_t)qt * XCH_FLOATS * 4 + 256 + 1024 + extra;
}

// `count` tiles of up to 256 queries; extra: bytes of the bias table.
template <class P>
int launch(Ctx* c, const P& p, const CUtensorMap& tm_a, const CUtensorMap& tm_b, int count, int nb_k, int nb_v, size_t extra) {
  Cfg cf;
  cf.nb_k = nb_k;
  cf.nb_v = nb_v;
  int qt = 2;
  cf.v_stages = 2;
  if (smem_bytes(nb_k, nb_v, 2, 2, extra) > kSmemMax) cf.v_stages = 1;
  if (smem_bytes(nb_k, nb_v, 2, cf.v_stages, extra) > kSmemMax) {
    qt = 1;
    cf.v_stages = 2;
  }
  const size_t smem = smem_bytes(nb_k, nb_v, qt, cf.v_stages, extra);
  RB_REQUIRE(smem <= kSmemMax, "attention: head sizes too large for the tcgen05 kernel");
  static bool attr_set = false;
  if (!attr_set) {
    RB_CUDA(cudaFuncSetAttribute(flash_tc_kernel<1, P>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemMax));
    RB_CUDA(cudaFuncSetAttribute(flash_tc_kernel<2, P>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemMax));
    attr_set = true;
  }
  if (qt == 2)
    RB_CUDA(launch_k(flash_tc_kernel<2, P>, dim3((unsigned)count, (unsigned)p.heads), dim3(64 + 2 * 256), smem, c->stream, c->use_pdl, tm_a, tm_b, p, cf));
  else
    RB_CUDA(launch_k(flash_tc_kernel<1, P>, dim3((unsigned)count * 2, (unsigned)p.heads), dim3(64 + 256), smem, c->stream, c->use_pdl, tm_a, tm_b, p, cf));
  ++g_launch_total;
  return REWB200_OK;
}

}  // namespace flash
}  // namespace rewb
