// Kernels of gqa_mix.cuh for any dtype and size.  Scores, softmax, mixing and gates are f32.
#include <math.h>

#include <algorithm>
#include <type_traits>

#include "act.cuh"
#include "gqa_mix.cuh"
#include "ptx.cuh"

namespace rewb {

extern int64_t g_launch_total;

namespace {

constexpr int PAGE_TOKENS = 64;
constexpr size_t PLAIN_WORK = (size_t)256 << 20;   // scratch of the plain kernels at most: larger steps run in pieces

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}

// The keys a query at `pos` sees, as a list: the kept first ones below its window, then the window.
struct Seen {
  int kept, lo, n;
};
__device__ __forceinline__ Seen seen_by(const GqaDims& m, int pos) {
  const int lo = m.window > 0 ? max(0, pos - m.window + 1) : 0, kept = min(m.keep_first, lo);
  return Seen{kept, lo, kept + pos - lo + 1};
}
__device__ __forceinline__ int seen_key(const Seen& s, int i) { return i < s.kept ? i : s.lo + i - s.kept; }

int64_t most_seen(const GqaDims& m, int64_t max_ctx) { return m.window > 0 ? std::min<int64_t>(max_ctx, (int64_t)m.window + m.keep_first) : max_ctx; }

// grid (rows of a piece, heads): the softmax weights of a row and head, [row][head][slots].
template <typename T>
__global__ void __launch_bounds__(128) mix_plain_weights_kernel(GqaMixArgs a, int64_t row0, int64_t slots) {
  extern __shared__ float q[];
  __shared__ float red[8];
  pdl_launch_dependents();
  pdl_wait();
  const int64_t row = row0 + blockIdx.x;
  const int h = blockIdx.y, K = a.m.dim, G = a.m.kv_heads, hk = h / (a.m.heads / G), w = threadIdx.x >> 5, ln = threadIdx.x & 31;
  const T* qp = reinterpret_cast<const T*>(a.q) + row * a.ldq + (int64_t)h * K;
  for (int i = threadIdx.x; i < K; i += 128) q[i] = ldf<T>(qp[i]);
  const int lane = row_lane(a.map, row), pos = min(max(row_pos(a.map, row), 0), a.max_pages * PAGE_TOKENS - 1);
  const Seen s = seen_by(a.m, pos);
  const float* tab = a.m.bias ? a.m.bias + (int64_t)h * a.m.n_bias : nullptr;
  float* p = a.work + ((int64_t)blockIdx.x * a.m.heads + h) * slots;
  __syncthreads();
  float mx = a.m.sink ? a.m.sink[h] : -INFINITY;
  for (int i = w; i < s.n; i += 4) {
    const int key = seen_key(s, i), page = a.block_table[(int64_t)lane * a.max_pages + key / PAGE_TOKENS];
    const T* kp = reinterpret_cast<const T*>(a.kc) + (((int64_t)page * G + hk) * PAGE_TOKENS + key % PAGE_TOKENS) * a.ldk;
    float z = 0.f;
    for (int j = ln; j < K; j += 32) z = fmaf(q[j], ldf<T>(kp[j]), z);
    z = warp_sum(z) * a.m.scale + (tab ? tab[min(pos - key, a.m.n_bias - 1)] : 0.f);
    mx = fmaxf(mx, z);
    if (ln == 0) p[i] = z;
  }
  if (ln == 0) red[w] = mx;
  __syncthreads();
  mx = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
  float l = 0.f;
  for (int i = threadIdx.x; i < s.n; i += 128) {
    const float e = expf(p[i] - mx);
    p[i] = e;
    l += e;
  }
  l = warp_sum(l);
  if (ln == 0) red[4 + w] = l;
  __syncthreads();
  l = (red[4] + red[5]) + (red[6] + red[7]);
  if (a.m.sink) l += expf(a.m.sink[h] - mx);
  const float inv = 1.0f / l;
  for (int i = threadIdx.x; i < s.n; i += 128) p[i] *= inv;   // the thread's own
}

// grid (rows of a piece, heads): mixed weights times values, gate.
template <typename T>
__global__ void __launch_bounds__(128) mix_plain_values_kernel(GqaMixArgs a, int64_t row0, int64_t slots) {
  constexpr int TILE = 128;
  __shared__ float wt[TILE];
  pdl_launch_dependents();
  pdl_wait();
  const int64_t row = row0 + blockIdx.x;
  const int h = blockIdx.y, H = a.m.heads, V = a.m.vdim, G = a.m.kv_heads, hk = h / (H / G);
  const int lane = row_lane(a.map, row), pos = min(max(row_pos(a.map, row), 0), a.max_pages * PAGE_TOKENS - 1);
  const Seen s = seen_by(a.m, pos);
  const float* p = a.work + (int64_t)blockIdx.x * H * slots;
  const float gh = a.gate_head ? a.gate_head[row * H + h] : 1.0f;
  for (int v0 = 0; v0 < V; v0 += 128) {
    const int v = v0 + threadIdx.x;
    float o = 0.f;
    for (int i0 = 0; i0 < s.n; i0 += TILE) {
      const int n = min(TILE, s.n - i0), i = threadIdx.x;
      if (i < n) {
        float z = 0.f;
        if (a.m.talk)
          for (int g = 0; g < H; ++g) z = fmaf(a.m.talk[(int64_t)h * H + g], p[(int64_t)g * slots + i0 + i], z);
        else
          z = p[(int64_t)h * slots + i0 + i];
        wt[i] = z;
      }
      __syncthreads();
      if (v < V)
        for (int j = 0; j < n; ++j) {
          const int key = seen_key(s, i0 + j), page = a.block_table[(int64_t)lane * a.max_pages + key / PAGE_TOKENS];
          o = fmaf(wt[j], ldf<T>(reinterpret_cast<const T*>(a.vc)[(((int64_t)page * G + hk) * PAGE_TOKENS + key % PAGE_TOKENS) * a.ldv + v]), o);
        }
      __syncthreads();
    }
    if (v >= V) continue;
    float g = gh * a.m.out_scale;
    if (a.gate) {
      float z = 0.f;
      for (int k = 0; k < a.nsplit; ++k) z += a.gate[k * a.split_stride + row * a.ld + (int64_t)h * V + v];
      g *= sigmoid_act(z);
    }
    reinterpret_cast<T*>(a.out)[row * a.ldo + (int64_t)h * V + v] = stf<T>(o * g);
  }
}

// ------------------------------------------------------------------ bf16 on the tensor cores
// Two launches over the pages a tile of rows sees (kept pages, then the window's), grid (splits, tiles * subtiles, kv heads *
// head groups), four consumer warps and a TMA warp; a CTA's 16 rows are `heads_per` query heads of one kv head times
// `tokens_per` tokens.
//   mix_scores_kernel   scores in base 2 (-inf where a query does not see the key) to scratch [row][head][slots], and the
//                       maximum and the sum of every row, head and split
//   mix_values_kernel   weights of all heads from them, mixed for this CTA's heads (f32), times the values
constexpr float LOG2E = 1.4426950408889634f;
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

struct MixCfg {
  int nb;             // 64-column boxes of a key or value row
  int stages;
  int heads_per, hgroups, tokens_per, subtiles;
  int splits;
  int tile0;          // first tile of this launch
  int64_t slots;
  float* s;           // scratch rows are tiles of the launch * max_tile_rows: [rows][heads][slots]
  float2* ml;         // [rows][heads][splits]
  float* o_part;      // [rows][heads][splits][vdim]
};

// The pages a tile sees.
struct Pages {
  int kept, w0, n;    // pages of kept keys below the window's first page, that page, all
  __device__ __forceinline__ int at(int i) const { return i < kept ? i : w0 + i - kept; }
};
__device__ __forceinline__ Pages pages_of(const GqaDims& m, int pos_first, int pos_last) {
  const int lo = m.window > 0 ? max(0, pos_first - m.window + 1) : 0, w0 = lo / PAGE_TOKENS;
  const int kept = min((m.keep_first + PAGE_TOKENS - 1) / PAGE_TOKENS, w0);
  return Pages{kept, w0, kept + pos_last / PAGE_TOKENS - w0 + 1};
}
int64_t most_pages(const GqaDims& m, int64_t tile_rows, int64_t max_pages) {
  if (m.window == 0) return max_pages;
  return std::min<int64_t>(max_pages, (m.keep_first + PAGE_TOKENS - 1) / PAGE_TOKENS + (m.window + tile_rows + PAGE_TOKENS - 3) / PAGE_TOKENS + 1);
}

// What a CTA works on.
struct CtaRows {
  int64_t row0, srow0;   // of the step, of the scratch
  int ntok, hk, head0, nh, lane, pos_first, pos_last, t0, nt;
  Pages pg;
};
__device__ __forceinline__ bool cta_rows(const GqaMixArgs& a, const MixCfg& cf, CtaRows& r) {
  const int2 tr = tile_rows(a.tiles, cf.tile0 + (int)blockIdx.y / cf.subtiles);
  const int tok0 = ((int)blockIdx.y % cf.subtiles) * cf.tokens_per, group = a.m.heads / a.m.kv_heads;
  r.ntok = min(cf.tokens_per, tr.y - tok0);
  if (r.ntok <= 0) return false;
  r.row0 = tr.x + tok0;
  r.srow0 = (int64_t)((int)blockIdx.y / cf.subtiles) * a.max_tile_rows + tok0;
  r.hk = blockIdx.z / cf.hgroups;
  const int hsub = ((int)blockIdx.z % cf.hgroups) * cf.heads_per;
  r.nh = min(cf.heads_per, group - hsub);
  r.head0 = r.hk * group + hsub;
  r.lane = row_lane(a.map, r.row0);
  const int cap = a.max_pages * PAGE_TOKENS;
  // the page list is the tile's, so that every subtile and both kernels count slots alike
  const int first = min(max(row_pos(a.map, tr.x), 0), cap - 1), last = min(first + tr.y - 1, cap - 1);
  r.pg = pages_of(a.m, first, last);
  r.pos_first = min(first + tok0, cap - 1);
  r.pos_last = last;
  const int per = (r.pg.n + cf.splits - 1) / cf.splits;
  r.t0 = (int)blockIdx.x * per;
  r.nt = max(0, min(per, r.pg.n - r.t0));
  return true;
}

// The TMA warp: pages t0 .. t0 + nt - 1 of the list through the ring.
__device__ __forceinline__ void load_pages(const GqaMixArgs& a, const MixCfg& cf, const CtaRows& r, const CUtensorMap& tm, uint8_t* ring, uint64_t* full,
                                           uint64_t* empty) {
  const int bytes = cf.nb * 8192;
  auto load = [&](int i) {
    const int st = i % cf.stages;
    const int y = (a.block_table[(int64_t)r.lane * a.max_pages + r.pg.at(r.t0 + i)] * a.m.kv_heads + r.hk) * PAGE_TOKENS;
    mbar_expect_tx(&full[st], bytes);
    for (int b = 0; b < cf.nb; ++b) tma_load_2d(ring + st * bytes + b * 8192, &tm, &full[st], b * 64, y);
  };
  int i = 0;
  if (a.early_kv) {
    for (; i < min(cf.stages, r.nt) && r.pg.at(r.t0 + i) < r.pos_last / PAGE_TOKENS; ++i) load(i);   // not the page the step writes
    pdl_wait();
  }
  for (; i < r.nt; ++i) {
    if (i >= cf.stages && !mbar_wait(&empty[i % cf.stages], ((i / cf.stages) - 1) & 1, a.status)) break;
    load(i);
  }
}
__device__ __forceinline__ void consumers_sync() { asm volatile("bar.sync 1, 128;" ::: "memory"); }

// KS: 16-feature steps of a key row.
template <int KS>
__global__ void __launch_bounds__(160, KS <= 8 ? 4 : 2) mix_scores_kernel(const __grid_constant__ CUtensorMap tm_k, GqaMixArgs a, MixCfg cf) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* sQ = smem + cf.stages * cf.nb * 8192;                    // [box][16 rows][128 bytes]
  float* sM = reinterpret_cast<float*>(sQ + cf.nb * 2048);          // [4 warps][16] maxima, [4][16] sums
  uint64_t *full = reinterpret_cast<uint64_t*>(sM + 128), *empty = full + 8;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l8 = lane & 7, lq = lane >> 3, g = lane >> 2, t = lane & 3;
  if (tid == 128) {
    for (int i = 0; i < cf.stages; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 4);
    }
    fence_barrier_init();
    tma_prefetch_desc(&tm_k);
  }
  pdl_launch_dependents();
  __syncthreads();
  if (!a.early_kv) pdl_wait();
  CtaRows r;
  if (!cta_rows(a, cf, r)) return;
  if (warp == 4) {
    if (lane == 0) load_pages(a, cf, r, tm_k, smem, full, empty);
    return;
  }
  if (a.early_kv) pdl_wait();
  for (int i = tid; i < 16 * cf.nb * 8; i += 128) {
    const int m = i / (cf.nb * 8), c = i % (cf.nb * 8), tok = m / cf.heads_per, hh = m % cf.heads_per;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (tok < r.ntok && hh < r.nh && c * 8 < a.m.dim)   // dim is a multiple of 8
      v = *reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(a.q) + (r.row0 + tok) * a.ldq + (int64_t)(r.head0 + hh) * a.m.dim + c * 8);
    *reinterpret_cast<uint4*>(sQ + (c >> 3) * 2048 + swz128((uint32_t)m, (uint32_t)(c & 7))) = v;
  }
  consumers_sync();
  const int ks = (a.m.dim + 15) / 16;
  uint32_t qf[KS][4];
  const uint32_t q_base = smem_u32(sQ);
#pragma unroll
  for (int k = 0; k < KS; ++k)
    if (k < ks)
      ldmatrix_x4(qf[k][0], qf[k][1], qf[k][2], qf[k][3], q_base + (k >> 2) * 2048 + swz128((lq & 1) * 8 + l8, (k & 3) * 2 + (lq >> 1)));
  // this thread's rows: g and g + 8
  const float sl2 = a.m.scale * LOG2E;
  int pos[2], low[2];
  float* sp[2];
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const int m = g + 8 * x, tok = m / cf.heads_per, hh = m % cf.heads_per;
    const bool on = tok < r.ntok && hh < r.nh;
    pos[x] = on ? r.pos_first + tok : -1;      // -1: sees no key
    low[x] = a.m.window > 0 ? pos[x] - a.m.window : -1;   // the key before the window
    sp[x] = on ? cf.s + ((r.srow0 + tok) * a.m.heads + r.head0 + hh) * cf.slots : nullptr;
  }
  float mrun[2] = {-INFINITY, -INFINITY}, lrun[2] = {0.f, 0.f};
  uint32_t k_off[4];
#pragma unroll
  for (int u = 0; u < 4; ++u) k_off[u] = swz128(warp * 16 + (lq >> 1) * 8 + l8, u * 2 + (lq & 1));
  const uint32_t ring = smem_u32(smem);
  bool ok = true;
  for (int it = 0; it < r.nt; ++it) {
    const int st = it % cf.stages;
    if (ok) ok = mbar_wait(&full[st], (it / cf.stages) & 1, a.status);
    const uint32_t kp = ring + st * cf.nb * 8192;
    float sc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
    for (int k = 0; k < KS; ++k) {
      if (k >= ks) break;
      uint32_t b0, b1, b2, b3;
      ldmatrix_x4(b0, b1, b2, b3, kp + (k >> 2) * 8192 + k_off[k & 3]);
      mma_bf16_16816(sc[0], qf[k], b0, b1);
      mma_bf16_16816(sc[1], qf[k], b2, b3);
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[st]);
    const int in_page = warp * 16 + 2 * t, key0 = r.pg.at(r.t0 + it) * PAGE_TOKENS + in_page;
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int x = e >> 1, key = key0 + n * 8 + (e & 1);
        sc[n][e] = key <= pos[x] && (key > low[x] || key < a.m.keep_first) ? sc[n][e] * sl2 : -INFINITY;
        mx[x] = fmaxf(mx[x], sc[n][e]);
      }
#pragma unroll
    for (int x = 0; x < 2; ++x) {
      if (sp[x]) {
        float* p = sp[x] + (int64_t)(r.t0 + it) * PAGE_TOKENS + in_page;
        *reinterpret_cast<float2*>(p) = make_float2(sc[0][2 * x], sc[0][2 * x + 1]);
        *reinterpret_cast<float2*>(p + 8) = make_float2(sc[1][2 * x], sc[1][2 * x + 1]);
      }
      const float mn = fmaxf(mrun[x], mx[x]), use = mn == -INFINITY ? 0.f : mn;   // a thread's own maximum: no exchange per page
      lrun[x] = lrun[x] * ex2(mrun[x] - use) + (ex2(sc[0][2 * x] - use) + ex2(sc[0][2 * x + 1] - use)) + (ex2(sc[1][2 * x] - use) + ex2(sc[1][2 * x + 1] - use));
      mrun[x] = mn;
    }
  }
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    float mn = mrun[x];
    mn = fmaxf(mn, __shfl_xor_sync(0xffffffffu, mn, 1));
    mn = fmaxf(mn, __shfl_xor_sync(0xffffffffu, mn, 2));
    lrun[x] *= ex2(mrun[x] - (mn == -INFINITY ? 0.f : mn));
    lrun[x] += __shfl_xor_sync(0xffffffffu, lrun[x], 1);
    lrun[x] += __shfl_xor_sync(0xffffffffu, lrun[x], 2);
    if (t == 0) {
      sM[warp * 16 + g + 8 * x] = mn;
      sM[64 + warp * 16 + g + 8 * x] = lrun[x];
    }
  }
  consumers_sync();
  if (tid < 16) {
    const int tok = tid / cf.heads_per, hh = tid % cf.heads_per;
    if (tok < r.ntok && hh < r.nh) {
      float M = -INFINITY, l = 0.f;
#pragma unroll
      for (int w = 0; w < 4; ++w) M = fmaxf(M, sM[w * 16 + tid]);
      const float use = M == -INFINITY ? 0.f : M;
#pragma unroll
      for (int w = 0; w < 4; ++w) l += ex2(sM[w * 16 + tid] - use) * sM[64 + w * 16 + tid];
      cf.ml[((r.srow0 + tok) * a.m.heads + r.head0 + hh) * cf.splits + blockIdx.x] = make_float2(M, l);
    }
  }
}

constexpr int LDP = 64 + 8;   // elements of a row of mixed weights

// VW: 16-column groups of a value row a warp has.
template <int VW>
__global__ void __launch_bounds__(160, VW <= 2 ? 4 : 2) mix_values_kernel(const __grid_constant__ CUtensorMap tm_v, GqaMixArgs a, MixCfg cf) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int H = a.m.heads, V = a.m.vdim;
  bf16* sP = reinterpret_cast<bf16*>(smem + cf.stages * cf.nb * 8192);    // [2][16][LDP] mixed weights
  float* sX = reinterpret_cast<float*>(sP + 2 * 16 * LDP);                // [heads_per][64] sums of the upper threads
  float* sT = sX + cf.heads_per * 64;                                     // [H][heads_per] mixing matrix
  float2* sN = reinterpret_cast<float2*>(sT + (H * cf.heads_per + 1) / 2 * 2);   // [tokens_per][H] maximum, 1 / sum
  uint64_t *full = reinterpret_cast<uint64_t*>(sN + cf.tokens_per * H), *empty = full + 8;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l8 = lane & 7, lq = lane >> 3, g = lane >> 2, t = lane & 3;
  if (tid == 128) {
    for (int i = 0; i < cf.stages; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 4);
    }
    fence_barrier_init();
    tma_prefetch_desc(&tm_v);
  }
  pdl_launch_dependents();
  __syncthreads();
  if (!a.early_kv) pdl_wait();
  CtaRows r;
  if (!cta_rows(a, cf, r)) return;
  if (warp == 4) {
    if (lane == 0) load_pages(a, cf, r, tm_v, smem, full, empty);
    return;
  }
  // the mixing matrix depends on no earlier kernel
  for (int i = tid; i < H * cf.heads_per; i += 128) {
    const int j = i / cf.heads_per, hh = i % cf.heads_per, h = r.head0 + hh;
    sT[i] = hh >= r.nh ? 0.f : a.m.talk ? a.m.talk[(int64_t)h * H + j] : j == h ? 1.f : 0.f;
  }
  for (int i = tid; i < 16 * LDP; i += 128) reinterpret_cast<uint32_t*>(sP)[i] = 0u;   // rows nobody writes
  if (a.early_kv) pdl_wait();
  for (int i = tid; i < r.ntok * H; i += 128) {
    const float2* e = cf.ml + ((r.srow0 + i / H) * H + i % H) * cf.splits;
    float M = -INFINITY, l = 0.f;
    for (int s = 0; s < cf.splits; ++s) M = fmaxf(M, e[s].x);
    const float use = M == -INFINITY ? 0.f : M;
    for (int s = 0; s < cf.splits; ++s) l += ex2(e[s].x - use) * e[s].y;
    sN[i] = make_float2(use, l > 0.f ? 1.0f / l : 0.f);
  }
  consumers_sync();
  float acc[VW][2][4];
#pragma unroll
  for (int j = 0; j < VW; ++j)
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[j][e >> 2][e & 3] = 0.f;
  const int vg = (V + 15) / 16, key = tid & 63, upper = tid >> 6;
  const uint32_t ring = smem_u32(smem);
  bool ok = true;
  for (int it = 0; it < r.nt; ++it) {
    const int st = it % cf.stages;
    bf16* const P = sP + (it & 1) * 16 * LDP;
    // ---- mixed weights of the page: a thread has a key, the two halves of the threads share the heads
    for (int tok = 0; tok < r.ntok; ++tok) {
      const float* s = cf.s + (r.srow0 + tok) * H * cf.slots + (int64_t)(r.t0 + it) * PAGE_TOKENS + key;
      const float2* nrm = sN + tok * H;
      float w[16];
#pragma unroll
      for (int hh = 0; hh < 16; ++hh) w[hh] = 0.f;
      auto mix = [&](auto n) {   // n: heads_per rounded up
        constexpr int N = decltype(n)::value;
#pragma unroll 8
        for (int j = upper; j < H; j += 2) {
          const float2 e = nrm[j];
          const float p = ex2(s[j * cf.slots] - e.x) * e.y;
          const float* T = sT + j * cf.heads_per;
#pragma unroll
          for (int hh = 0; hh < N; ++hh)
            if (hh < cf.heads_per) w[hh] = fmaf(T[hh], p, w[hh]);
        }
        if (upper)
#pragma unroll
          for (int hh = 0; hh < N; ++hh)
            if (hh < cf.heads_per) sX[hh * 64 + key] = w[hh];
        consumers_sync();
        if (!upper)
#pragma unroll
          for (int hh = 0; hh < N; ++hh)
            if (hh < cf.heads_per) P[(tok * cf.heads_per + hh) * LDP + key] = __float2bfloat16_rn(w[hh] + sX[hh * 64 + key]);
      };
      if (cf.heads_per <= 4) mix(std::integral_constant<int, 4>{});
      else if (cf.heads_per <= 8) mix(std::integral_constant<int, 8>{});
      else mix(std::integral_constant<int, 16>{});
      consumers_sync();
    }
    if (ok) ok = mbar_wait(&full[st], (it / cf.stages) & 1, a.status);
    // ---- times values: a warp has its columns of all keys
    const uint32_t vp = ring + st * cf.nb * 8192, pa = smem_u32(P) + (((lq & 1) * 8 + l8) * LDP + (lq >> 1) * 8) * 2;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      uint32_t pf[4];
      ldmatrix_x4(pf[0], pf[1], pf[2], pf[3], pa + k * 32);
#pragma unroll
      for (int j = 0; j < VW; ++j) {
        const int c = warp * VW + j;
        if (c >= vg) break;
        uint32_t v0, v1, v2, v3;
        ldmatrix_x4_trans(v0, v1, v2, v3, vp + (c >> 2) * 8192 + swz128(k * 16 + (lq & 1) * 8 + l8, (c & 3) * 2 + (lq >> 1)));
        mma_bf16_16816(acc[j][0], pf, v0, v1);
        mma_bf16_16816(acc[j][1], pf, v2, v3);
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[st]);
  }
#pragma unroll
  for (int x = 0; x < 2; ++x) {
    const int m = g + 8 * x, tok = m / cf.heads_per, hh = m % cf.heads_per;
    if (tok >= r.ntok || hh >= r.nh) continue;
    const int64_t row = r.row0 + tok;
    const int h = r.head0 + hh;
    const float gh = (a.gate_head ? a.gate_head[row * H + h] : 1.0f) * a.m.out_scale;
#pragma unroll
    for (int j = 0; j < VW; ++j)
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const int col = (warp * VW + j) * 16 + n * 8 + 2 * t;
        if (col >= V) continue;   // vdim is a multiple of 8
        float2 o = make_float2(acc[j][n][2 * x], acc[j][n][2 * x + 1]);
        if (cf.splits > 1) {
          *reinterpret_cast<float2*>(cf.o_part + (((r.srow0 + tok) * H + h) * cf.splits + blockIdx.x) * V + col) = o;
          continue;
        }
        float2 ge = make_float2(gh, gh);
        if (a.gate) {
          const float* z = a.gate + row * a.ld + (int64_t)h * V + col;
          float z0 = 0.f, z1 = 0.f;
          for (int k = 0; k < a.nsplit; ++k) {
            z0 += z[k * a.split_stride];
            z1 += z[k * a.split_stride + 1];
          }
          ge.x *= sigmoid_act(z0);
          ge.y *= sigmoid_act(z1);
        }
        *reinterpret_cast<uint32_t*>(reinterpret_cast<bf16*>(a.out) + row * a.ldo + (int64_t)h * V + col) = pack_bf16(o.x * ge.x, o.y * ge.y);
      }
  }
}

// One warp per (row of a tile, head): sums the splits, applies the gate.
__global__ void __launch_bounds__(256) mix_merge_kernel(GqaMixArgs a, MixCfg cf, int64_t units) {
  pdl_launch_dependents();
  const int64_t u = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int ln = threadIdx.x & 31, H = a.m.heads, V = a.m.vdim;
  if (u >= units) return;
  pdl_wait();
  const int64_t slot = u / H;
  const int h = (int)(u % H);
  const int2 tr = tile_rows(a.tiles, cf.tile0 + (int)(slot / a.max_tile_rows));
  const int k = (int)(slot % a.max_tile_rows);
  if (k >= tr.y) return;
  const int64_t row = tr.x + k;
  const float* p = cf.o_part + (slot * H + h) * cf.splits * V;
  const float gh = (a.gate_head ? a.gate_head[row * H + h] : 1.0f) * a.m.out_scale;
  for (int c = ln * 4; c < V; c += 128) {
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int s = 0; s < cf.splits; ++s) {
      const float4 x = *reinterpret_cast<const float4*>(p + s * V + c);
      o.x += x.x; o.y += x.y; o.z += x.z; o.w += x.w;
    }
    float4 ge = make_float4(gh, gh, gh, gh);
    if (a.gate) {
      float e[4] = {0.f, 0.f, 0.f, 0.f};
      const float* z = a.gate + row * a.ld + (int64_t)h * V + c;
      for (int s = 0; s < a.nsplit; ++s)
#pragma unroll
        for (int x = 0; x < 4; ++x) e[x] += z[s * a.split_stride + x];
      ge = make_float4(gh * sigmoid_act(e[0]), gh * sigmoid_act(e[1]), gh * sigmoid_act(e[2]), gh * sigmoid_act(e[3]));
    }
    *reinterpret_cast<uint2*>(reinterpret_cast<bf16*>(a.out) + row * a.ldo + (int64_t)h * V + c) =
        make_uint2(pack_bf16(o.x * ge.x, o.y * ge.y), pack_bf16(o.z * ge.z, o.w * ge.w));
  }
}

bool mma_ok(const GqaDims& m) {
  return m.dim % 8 == 0 && m.vdim % 8 == 0 && m.dim <= 256 && m.vdim <= 256 && !m.bias && !m.sink && m.heads <= 256;
}

MixCfg config(const GqaDims& m, int max_tile_rows) {
  MixCfg cf = {};
  const int group = m.heads / m.kv_heads;
  cf.heads_per = std::min(group, 16);
  cf.hgroups = (group + cf.heads_per - 1) / cf.heads_per;
  cf.tokens_per = std::min(max_tile_rows, std::max(1, 16 / cf.heads_per));
  cf.subtiles = (max_tile_rows + cf.tokens_per - 1) / cf.tokens_per;
  return cf;
}
int splits_of(Ctx* c, const GqaDims& m, const MixCfg& cf, int64_t tiles, int64_t pages) {
  const int64_t ctas = std::max<int64_t>(1, tiles * cf.subtiles * m.kv_heads * cf.hgroups);
  return (int)std::max<int64_t>(1, std::min<int64_t>({(3 * c->sm_count + ctas - 1) / ctas, pages, 16}));
}
size_t row_bytes(const GqaDims& m, int64_t slots, int splits) {
  return (size_t)m.heads * (slots * sizeof(float) + splits * sizeof(float2) + (splits > 1 ? (size_t)splits * m.vdim * sizeof(float) : 0));
}
constexpr size_t MIX_WORK = (size_t)256 << 20;

}  // namespace

size_t gqa_mix_bytes(Ctx* c, const GqaDims& m, int dtype, int64_t rows, int64_t tiles, int64_t max_tile_rows, int64_t max_ctx) {
  const size_t row = (size_t)m.heads * most_seen(m, max_ctx) * sizeof(float);
  const size_t plain = std::max(row, std::min(PLAIN_WORK, row * (size_t)rows));
  if (dtype != REWB200_BF16 || !mma_ok(m)) return plain;
  const MixCfg cf = config(m, (int)max_tile_rows);
  const int64_t pages = most_pages(m, max_tile_rows, (max_ctx + PAGE_TOKENS - 1) / PAGE_TOKENS);
  const size_t per = row_bytes(m, pages * PAGE_TOKENS, splits_of(c, m, cf, tiles, pages));
  return std::max(plain, std::max(per * (size_t)max_tile_rows, std::min(MIX_WORK, per * (size_t)(tiles * max_tile_rows))));
}

namespace {

int plain_launch(Ctx* c, const GqaMixArgs& a) {
  const int64_t slots = most_seen(a.m, (int64_t)a.max_pages * PAGE_TOKENS);
  const int64_t piece = std::min<int64_t>(a.rows, (int64_t)(a.work_bytes / ((size_t)a.m.heads * slots * sizeof(float))));
  RB_REQUIRE(piece > 0 || a.rows == 0, "attention with mixed heads: scratch too small");
  const bool bf = a.dtype == REWB200_BF16;
  for (int64_t r = 0; r < a.rows; r += piece) {
    const dim3 grid((unsigned)std::min(piece, a.rows - r), (unsigned)a.m.heads);
    const size_t smem = (size_t)a.m.dim * sizeof(float);
    RB_CUDA(bf ? launch_k(mix_plain_weights_kernel<bf16>, grid, dim3(128), smem, c->stream, c->use_pdl, a, r, slots)
               : launch_k(mix_plain_weights_kernel<float>, grid, dim3(128), smem, c->stream, c->use_pdl, a, r, slots));
    RB_CUDA(bf ? launch_k(mix_plain_values_kernel<bf16>, grid, dim3(128), (size_t)0, c->stream, c->use_pdl, a, r, slots)
               : launch_k(mix_plain_values_kernel<float>, grid, dim3(128), (size_t)0, c->stream, c->use_pdl, a, r, slots));
    g_launch_total += 2;
  }
  return REWB200_OK;
}

}  // namespace

int gqa_mix_launch(Ctx* c, const GqaMixArgs& a) {
  if (a.tiles.count == 0) return REWB200_OK;
  if (a.dtype != REWB200_BF16 || c->gqa_impl == 1 || !mma_ok(a.m)) return plain_launch(c, a);
  MixCfg cf = config(a.m, a.max_tile_rows);
  const int64_t pages = most_pages(a.m, a.max_tile_rows, a.max_pages);
  cf.slots = pages * PAGE_TOKENS;
  cf.splits = splits_of(c, a.m, cf, a.tiles.count, pages);
  const size_t per = row_bytes(a.m, cf.slots, cf.splits);
  const int64_t room = (int64_t)(a.work_bytes / per);        // rows a piece may have
  const int64_t piece = room / a.max_tile_rows;              // ... and tiles
  RB_REQUIRE(piece > 0, "attention with mixed heads: scratch too small");
  const int ks = (a.m.dim + 15) / 16, vg = (a.m.vdim + 15) / 16;
  auto go = [&](auto kernel, const CUtensorMap& tm, size_t smem, dim3 grid) -> int {
    if (smem > 48 * 1024) RB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    RB_CUDA(launch_k(kernel, grid, dim3(160), smem, c->stream, c->use_pdl, tm, a, cf));
    ++g_launch_total;
    return REWB200_OK;
  };
  for (int64_t t0 = 0; t0 < a.tiles.count; t0 += piece) {
    const int64_t n = std::min<int64_t>(piece, a.tiles.count - t0);
    cf.tile0 = (int)t0;
    // in this order every part starts on 16 bytes: vdim is a multiple of 8, slots one of 64
    cf.o_part = a.work;
    cf.s = a.work + (cf.splits > 1 ? (size_t)room * a.m.heads * cf.splits * a.m.vdim : 0);
    cf.ml = reinterpret_cast<float2*>(cf.s + (size_t)room * a.m.heads * cf.slots);
    const dim3 grid((unsigned)cf.splits, (unsigned)(n * cf.subtiles), (unsigned)(a.m.kv_heads * cf.hgroups));
    cf.nb = (a.m.dim + 63) / 64;
    cf.stages = cf.nb <= 2 ? 3 : 2;
    size_t smem = (size_t)cf.stages * cf.nb * 8192 + cf.nb * 2048 + 512 + 128 + 1024;
    RB_TRY(ks <= 4 ? go(mix_scores_kernel<4>, *a.tm_k, smem, grid) : ks <= 8 ? go(mix_scores_kernel<8>, *a.tm_k, smem, grid) : go(mix_scores_kernel<16>, *a.tm_k, smem, grid));
    cf.nb = (a.m.vdim + 63) / 64;
    cf.stages = 2;
    smem = (size_t)cf.stages * cf.nb * 8192 + 2 * 16 * LDP * 2 + (size_t)cf.heads_per * 64 * 4 + ((size_t)a.m.heads * cf.heads_per + 1) / 2 * 8 +
           (size_t)cf.tokens_per * a.m.heads * 8 + 128 + 1024;
    RB_TRY(vg <= 4 ? go(mix_values_kernel<1>, *a.tm_v, smem, grid) : vg <= 8 ? go(mix_values_kernel<2>, *a.tm_v, smem, grid) : go(mix_values_kernel<4>, *a.tm_v, smem, grid));
    if (cf.splits > 1) {
      const int64_t units = n * a.max_tile_rows * a.m.heads;
      RB_CUDA(launch_k(mix_merge_kernel, dim3((unsigned)((units + 7) / 8)), dim3(256), 0, c->stream, c->use_pdl, a, cf, units));
      ++g_launch_total;
    }
  }
  return REWB200_OK;
}

}  // namespace rewb
