// Gated linear attention of large prompt portions, in chunks of 32 tokens on the tensor cores.
//
// With b_t the running sum of the log decays of a key channel and r its value in the middle of the chunk,
//   q~_t = q_t e^(b_t - r)      k~_s = k_s e^(r - b_s)      A_ts = q~_t . k~_s  (s <= t)
//   o_t  = q~_t (e^r S) + sum_s A_ts v_s                    S <- e^(b_end - r) (e^r S + sum_s k~_s v_s^T)
// so one pair of scaled operands serves the scores, the output and the state.  Two launches:
//   gla_prepare_kernel   one CTA per chunk and head: decays, q~, k~, v, A and the decays of the two halves, as one block in
//                        the layout the second kernel has in shared memory (one bulk store)
//   gla_scan_kernel      one CTA walks the chunks of a portion for one head (or for a slice of its value columns; a cluster
//                        shares the head): blocks arrive by bulk copies two chunks ahead, the state stays in registers.
//                        Warp w holds the transposed state [16 value rows][dim], whose accumulator fragments are also the
//                        A operand of q~ S.
// Decays, their sums and the state are f32; operands of products are bf16 (the state as a high part and a remainder) and
// sums f32.
//
// The two halves of a chunk bound the exponents: if a channel decays by more than 2^MAX_DECAY in one of them, the
// chunk runs token by token on the same registers.
#include <cooperative_groups.h>
#include <math.h>

#include <algorithm>

#include "gla.cuh"
#include "ptx.cuh"

namespace cg = cooperative_groups;

namespace rewb {

extern int64_t g_launch_total;

namespace {

constexpr int C = 32;             // tokens of a chunk
constexpr int NT = 256;
constexpr float MAX_DECAY = 50.f;
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void ldmatrix_x2(uint32_t& r0, uint32_t& r1, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
// -log2(sigmoid(z)): log1p of a small argument by its series, where 1 + u would round it away
__device__ __forceinline__ float neg_log2_sigmoid(float z) {
  const float u = ex2(-LOG2E * fabsf(z));
  float l;
  asm("lg2.approx.ftz.f32 %0, %1;" : "=f"(l) : "f"(1.0f + u));
  const float series = u * LOG2E * fmaf(u, fmaf(u, 0.33333333f, -0.5f), 1.0f);
  return fmaf(fmaxf(-z, 0.f), LOG2E, u < 0.015625f ? series : l);
}
// x, y = hi + lo, packed bf16 pairs
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(x, y);
  const __nv_bfloat162 h = *reinterpret_cast<const __nv_bfloat162*>(&hi);
  lo = pack_bf16(x - __low2float(h), y - __high2float(h));
}
__device__ __forceinline__ void bulk_store_1d(void* dst, const void* src, uint32_t bytes) {
  asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(dst), "r"(smem_u32(src)), "r"(bytes) : "memory");
  asm volatile("cp.async.bulk.commit_group;" ::: "memory");
}
// the source of this thread's bulk stores may be overwritten (or cease to exist) afterwards
__device__ __forceinline__ void bulk_store_wait() { asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory"); }

// The block of one chunk and head (byte offsets), rows padded by 16 bytes so that ldmatrix meets no bank conflicts.
struct ChunkLayout {
  int kt;        // 16-channel steps of a key: dim padded to 16 kt
  int vp;        // value columns, padded to a multiple of 16
  int ldq, ldv;  // elements of a q~ / k~ row and of a value row
  int k, v, a;   // q~ [C][ldq] at 0, k~ [C][ldq], values [C][ldv], A [C][C + 8]
  int f;         // decay up to the middle [16 kt], decay after it [16 kt]
  int far;       // 1: the chunk needs the token-by-token path
  int bytes;
};
constexpr int LDA = C + 8;

__host__ ChunkLayout layout_of(const GlaDims& m) {
  ChunkLayout c;
  c.kt = (m.dim + 15) / 16;
  c.vp = (m.vdim + 15) / 16 * 16;
  c.ldq = c.kt * 16 + 8;
  c.ldv = c.vp + 8;
  c.k = C * c.ldq * 2;
  c.v = c.k + C * c.ldq * 2;
  c.a = c.v + C * c.ldv * 2;
  c.f = c.a + C * LDA * 2;
  c.far = c.f + 2 * c.kt * 16 * 4;
  c.bytes = (c.far + 16 + 127) / 128 * 128;
  return c;
}

// grid (heads, chunks)
__global__ void __launch_bounds__(NT, 3) gla_prepare_kernel(GlaArgs a, ChunkLayout cl) {
  extern __shared__ __align__(128) uint8_t smem[];
  const GlaDims& m = a.m;
  const int K = m.dim, V = m.vdim, Kp = cl.kt * 16, rp = (m.rank + 3) / 4 * 4, ldq = cl.ldq, ldv = cl.ldv, ld = (int)a.ld;
  bf16* sQ = reinterpret_cast<bf16*>(smem);
  bf16* sK = reinterpret_cast<bf16*>(smem + cl.k);
  bf16* sV = reinterpret_cast<bf16*>(smem + cl.v);
  bf16* sA = reinterpret_cast<bf16*>(smem + cl.a);
  float* sF = reinterpret_cast<float*>(smem + cl.f);
  float* sA1 = reinterpret_cast<float*>(smem + cl.bytes);      // decay features, see a1_at
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l8 = lane & 7, lq = lane >> 3, g = lane >> 2, t4 = lane & 3;
  const int h = blockIdx.x, HK = m.heads * K, HV = m.heads * V;
  // this thread's pair of key channels and eight tokens: a warp has 32 channels of one half of the chunk, its upper lanes
  // the later eight tokens
  const int half = warp >> 2, kc = (warp & 3) * 32 + (lane & 15) * 2, late = lane >> 4, tb = half * 16 + late * 8;
  const bool mine = kc < Kp, live = kc < K;
  const uint32_t pair = __ballot_sync(0xffffffffu, mine);      // both lanes of a channel pair are in or out together
  // rows of decay features, with a gap every eight of them so that the two groups of lanes read different banks
  auto a1_at = [rp](int t, int r) { return t * rp + (t >> 3) * 4 + r; };
  pdl_launch_dependents();
  pdl_wait();
  const int2 ch = a.chunks[blockIdx.y];                         // first row, tokens
  const int nt = ch.y;
  const float* base = a.partial + (int64_t)ch.x * a.ld;
  for (int i = tid; i < C * rp; i += NT) {
    const int t = i / rp, r = i - t * rp;
    float v = 0.f;
    if (t < nt && r < m.rank)
      for (int s = 0; s < a.nsplit; ++s) v += base[s * a.split_stride + t * ld + 2 * HK + 2 * HV + r];
    sA1[a1_at(t, r)] = v;
  }
  // values: one group of four columns, tokens vt, vt + vstep, ..
  {
    const int vq = cl.vp / 4, vt = tid / vq, vc = (tid - vt * vq) * 4, vstep = NT / vq;
    const float* b = base + vt * ld + 2 * HK + h * V + vc;
    float4 x[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (vt < vstep && vt + i * vstep < nt && vc < V) x[i] = *reinterpret_cast<const float4*>(b + i * vstep * ld);
    }
    for (int s = 1; s < a.nsplit; ++s)
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (vt < vstep && vt + i * vstep < nt && vc < V) {
          const float4 w = *reinterpret_cast<const float4*>(b + s * a.split_stride + i * vstep * ld);
          x[i].x += w.x; x[i].y += w.y; x[i].z += w.z; x[i].w += w.w;
        }
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (vt < vstep && vt + i * vstep < C)
        *reinterpret_cast<uint2*>(sV + (vt + i * vstep) * ldv + vc) = make_uint2(pack_bf16(x[i].x, x[i].y), pack_bf16(x[i].z, x[i].w));
  }
  __syncthreads();
  bool far = false;
  if (mine) {
    const float* qp = base + tb * ld + h * K + kc;
    const int nu = live ? nt - tb : 0;
    auto rows8 = [&](const float* x, float2 (&y)[8]) {
      if (nu >= 8 && a.nsplit == 1) {
#pragma unroll
        for (int u = 0; u < 8; ++u) y[u] = *reinterpret_cast<const float2*>(x + u * ld);
        return;
      }
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        y[u] = make_float2(0.f, 0.f);
        if (u < nu)
          for (int s = 0; s < a.nsplit; ++s) {
            const float2 w = *reinterpret_cast<const float2*>(x + s * a.split_stride + u * ld);
            y[u].x += w.x;
            y[u].y += w.y;
          }
      }
    };
    float2 q[8], k[8], e[8];
    rows8(qp, q);
    rows8(qp + HK, k);
    const float2 kbias = live ? *reinterpret_cast<const float2*>(m.a2_b + h * K + kc) : make_float2(0.f, 0.f);
#pragma unroll
    for (int u = 0; u < 8; ++u) e[u] = kbias;
    const float* a2 = m.a2 + h * K + (live ? kc : 0);
    for (int r = 0; r < rp; r += 4) {
      float2 w[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) w[i] = *reinterpret_cast<const float2*>(a2 + min(r + i, m.rank - 1) * HK);   // features past rank are zero
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        const float4 x = *reinterpret_cast<const float4*>(sA1 + a1_at(tb + u, r));
        e[u].x = fmaf(x.x, w[0].x, fmaf(x.y, w[1].x, fmaf(x.z, w[2].x, fmaf(x.w, w[3].x, e[u].x))));
        e[u].y = fmaf(x.x, w[0].y, fmaf(x.y, w[1].y, fmaf(x.z, w[2].y, fmaf(x.w, w[3].y, e[u].y))));
      }
    }
    // log2 of the decays, then their sums from the middle of the chunk
    const float dscale = -1.0f / m.tau, qscale = rsqrtf((float)K);
    float2 part = make_float2(0.f, 0.f);
#pragma unroll
    for (int u = 0; u < 8; ++u) {
      e[u].x = neg_log2_sigmoid(e[u].x) * dscale;
      e[u].y = neg_log2_sigmoid(e[u].y) * dscale;
      if (u >= nu) e[u] = make_float2(0.f, 0.f);
      part.x += e[u].x;
      part.y += e[u].y;
    }
    const float2 other = make_float2(__shfl_xor_sync(pair, part.x, 16), __shfl_xor_sync(pair, part.y, 16));
    const float2 tot = make_float2(part.x + other.x, part.y + other.y);
    far = fminf(tot.x, tot.y) < -MAX_DECAY;
    if (!late) *reinterpret_cast<float2*>(sF + half * Kp + kc) = make_float2(ex2(tot.x), ex2(tot.y));
    // first half: minus the decays still ahead of the middle; second half: the decays since
    float2 run = half ? (late ? other : make_float2(0.f, 0.f)) : (late ? part : tot);
    bf16* dq = sQ + tb * ldq + kc;
    bf16* dk = sK + tb * ldq + kc;
#pragma unroll
    for (int u = 0; u < 8; ++u) {
      float2 b;
      if (half) {
        run.x += e[u].x;
        run.y += e[u].y;
        b = run;
      } else {
        run.x -= e[u].x;
        run.y -= e[u].y;
        b = make_float2(-run.x, -run.y);
      }
      if (far) b = make_float2(0.f, 0.f);
      *reinterpret_cast<uint32_t*>(dq + u * ldq) = pack_bf16(q[u].x * (qscale * ex2(b.x)), q[u].y * (qscale * ex2(b.y)));
      *reinterpret_cast<uint32_t*>(dk + u * ldq) = pack_bf16(k[u].x * ex2(-b.x), k[u].y * ex2(-b.y));
    }
  }
  const int any_far = __syncthreads_or(far ? 1 : 0);
  // scores: six 16 x 8 tiles on and below the diagonal (the scan never reads the block above it)
  if (warp < 6) {
    const int mt = warp < 2 ? 0 : 1, nn = warp < 2 ? warp : warp - 2;
    float s[4] = {0.f, 0.f, 0.f, 0.f};
    const uint32_t qa = smem_u32(sQ) + ((mt * 16 + (lq & 1) * 8 + l8) * ldq + (lq >> 1) * 8) * 2;
    const uint32_t ka = smem_u32(sK) + ((nn * 8 + l8) * ldq + (lq & 1) * 8) * 2;
#pragma unroll 4
    for (int k = 0; k < cl.kt; ++k) {
      uint32_t q[4], b0, b1;
      ldmatrix_x4(q[0], q[1], q[2], q[3], qa + k * 32);
      ldmatrix_x2(b0, b1, ka + k * 32);
      mma_bf16_16816(s, q, b0, b1);
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = mt * 16 + g + 8 * r, sc = nn * 8 + 2 * t4;
      *reinterpret_cast<uint32_t*>(sA + t * LDA + sc) = pack_bf16(sc <= t ? s[2 * r] : 0.f, sc + 1 <= t ? s[2 * r + 1] : 0.f);
    }
  }
  if (tid == NT - 1) *reinterpret_cast<int*>(smem + cl.far) = any_far;
  fence_proxy_async();
  __syncthreads();
  if (tid == 0) {
    bulk_store_1d(a.work + ((int64_t)blockIdx.y * m.heads + h) * cl.bytes, smem, (uint32_t)cl.bytes);
    bulk_store_wait();
  }
}

// grid (value slices, heads, portions), a warp per 16 value columns.  KT: capacity of the register state in 16-channel steps;
// vs: value columns of the CTA, a multiple of 16.
template <int KT, bool CLUSTER>
__global__ void __launch_bounds__(CLUSTER ? NT / 2 : NT, CLUSTER ? 3 : 2) gla_scan_kernel(GlaArgs a, ChunkLayout cl, int vs) {
  extern __shared__ __align__(128) uint8_t smem[];
  const GlaDims& m = a.m;
  const int K = m.dim, V = m.vdim, Kp = cl.kt * 16, ldq = cl.ldq, ldv = cl.ldv, ldO = vs + 4, ld = (int)a.ld;
  float* sO = reinterpret_cast<float*>(smem + 2 * cl.bytes);                 // [2][C][ldO]
  float* sS = sO + 2 * C * ldO;                                              // [2][C] sums of squares, [C] norms, [2][8 warps][C] sums of squares
  float* sX = sS + 3 * C + 2 * 8 * C;                                        // [3][Kp] q, k, alpha of a token (token-by-token path)
  uint64_t* full = reinterpret_cast<uint64_t*>(sX + 3 * Kp);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l8 = lane & 7, lq = lane >> 3, g = lane >> 2, t4 = lane & 3;
  const int h = blockIdx.y, v0 = blockIdx.x * vs, HK = m.heads * K, HV = m.heads * V;
  const int nthreads = 2 * vs;                                               // the block
  if (tid == 0) {
    mbar_init(full, 1);
    mbar_init(full + 1, 1);
    fence_barrier_init();
  }
  pdl_launch_dependents();
  __syncthreads();
  pdl_wait();
  const GlaPortion p = a.list[blockIdx.z];
  const int chunks = (p.n + C - 1) / C;
  auto load = [&](int c) {
    mbar_expect_tx(full + (c & 1), (uint32_t)cl.bytes);
    bulk_load_1d(smem + (c & 1) * cl.bytes, a.work + ((int64_t)(p.chunk0 + c) * m.heads + h) * cl.bytes, (uint32_t)cl.bytes, full + (c & 1));
  };
  if (tid == 0)
    for (int c = 0; c < min(2, chunks); ++c) load(c);
  float* const st = a.state + ((int64_t)p.lane * m.heads + h) * K * a.ldv;
  // S[j][e]: value row v0 + 16 warp + g + 8 (e >> 1), channel 8 j + 2 t4 + (e & 1)
  float S[2 * KT][4];
#pragma unroll
  for (int j = 0; j < 2 * KT; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int v = v0 + warp * 16 + g + 8 * (e >> 1), k = 8 * j + 2 * t4 + (e & 1);
      S[j][e] = p.pos0 > 0 && v < V && k < K ? st[k * a.ldv + v] : 0.f;
    }
  auto scale_state = [&](const float* f) {
#pragma unroll
    for (int j = 0; j < 2 * KT; ++j) {
      if (j >= 2 * cl.kt) break;
      const float2 x = *reinterpret_cast<const float2*>(f + j * 8 + 2 * t4);
      S[j][0] *= x.x;
      S[j][1] *= x.y;
      S[j][2] *= x.x;
      S[j][3] *= x.y;
    }
  };
  // output: one group of four columns, tokens vt, vt + vstep, ..
  constexpr int vstep = 8;   // 2 vs threads, vs / 4 column groups
  const int vq = vs / 4, vt = tid / vq, vc = (tid - vt * vq) * 4;
  const bool writes = v0 + vc < V;
  const float inv_v = 1.0f / (float)V;
  const int ldo = (int)a.ldo;
  bool ok = true;
  for (int it = 0; it < chunks; ++it) {
    const int nt = min(C, p.n - it * C);
    uint8_t* const blk = smem + (it & 1) * cl.bytes;
    const float* const base = a.partial + (int64_t)(p.row0 + it * C) * a.ld;
    float* const o_buf = sO + (it & 1) * C * ldO;
    float* const ss_buf = sS + 3 * C + (it & 1) * 8 * C;
    // the gates of the chunk are requested ahead of its products
    float4 gz[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      gz[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (writes && vt + i * vstep < nt) gz[i] = *reinterpret_cast<const float4*>(base + (vt + i * vstep) * ld + 2 * HK + HV + h * V + v0 + vc);
    }
    for (int s = 1; s < a.nsplit; ++s)
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (writes && vt + i * vstep < nt) {
          const float4 w = *reinterpret_cast<const float4*>(base + s * a.split_stride + (vt + i * vstep) * ld + 2 * HK + HV + h * V + v0 + vc);
          gz[i].x += w.x; gz[i].y += w.y; gz[i].z += w.z; gz[i].w += w.w;
        }
    if (ok) ok = mbar_wait(full + (it & 1), (it >> 1) & 1, a.status);
    if (*reinterpret_cast<const int*>(blk + cl.far) == 0) {
      {
        const uint32_t aQ = smem_u32(blk), aK = aQ + cl.k, aV = aQ + cl.v, aA = aQ + cl.a;
        const float* f = reinterpret_cast<const float*>(blk + cl.f);
        // (a slice has registers for a second set of sums: two shorter chains of products)
        float o[4][4], o2[4][4];
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
          for (int e = 0; e < 4; ++e) o[j][e] = o2[j][e] = 0.f;
        float(&ol)[4][4] = CLUSTER ? o2 : o;
        // ---- the state as every earlier token left it: o^T [16 value rows][C] = (e^r S)^T q~^T
        const uint32_t qb = aQ + (((lq >> 1) * 8 + l8) * ldq + (lq & 1) * 8) * 2, qb2 = qb + 16 * ldq * 2;
#pragma unroll
        for (int k = 0; k < KT; ++k) {
          if (k >= cl.kt) break;
          const float2 f0 = *reinterpret_cast<const float2*>(f + k * 16 + 2 * t4), f1 = *reinterpret_cast<const float2*>(f + k * 16 + 8 + 2 * t4);
          uint32_t sh[4], sl[4];
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            S[2 * k][2 * r] *= f0.x;
            S[2 * k][2 * r + 1] *= f0.y;
            S[2 * k + 1][2 * r] *= f1.x;
            S[2 * k + 1][2 * r + 1] *= f1.y;
            split2(S[2 * k][2 * r], S[2 * k][2 * r + 1], sh[r], sl[r]);
            split2(S[2 * k + 1][2 * r], S[2 * k + 1][2 * r + 1], sh[2 + r], sl[2 + r]);
          }
          uint32_t b[4], c[4];
          ldmatrix_x4(b[0], b[1], b[2], b[3], qb + k * 32);
          ldmatrix_x4(c[0], c[1], c[2], c[3], qb2 + k * 32);
          mma_bf16_16816(o[0], sh, b[0], b[1]);
          mma_bf16_16816(o[1], sh, b[2], b[3]);
          mma_bf16_16816(o[2], sh, c[0], c[1]);
          mma_bf16_16816(o[3], sh, c[2], c[3]);
          mma_bf16_16816(ol[0], sl, b[0], b[1]);
          mma_bf16_16816(ol[1], sl, b[2], b[3]);
          mma_bf16_16816(ol[2], sl, c[0], c[1]);
          mma_bf16_16816(ol[3], sl, c[2], c[3]);
        }
        // ---- o^T += v^T A^T, S^T += v^T k~, then the decay after the middle
        const uint32_t ab = aA + (((lq >> 1) * 8 + l8) * LDA + (lq & 1) * 8) * 2;
        const uint32_t kb = aK + (((lq & 1) * 8 + l8) * ldq + (lq >> 1) * 8) * 2;
#pragma unroll
        for (int s = 0; s < 2; ++s) {
          uint32_t vf[4];
          ldmatrix_x4_trans(vf[0], vf[1], vf[2], vf[3], aV + ((s * 16 + (lq >> 1) * 8 + l8) * ldv + v0 + warp * 16 + (lq & 1) * 8) * 2);
#pragma unroll
          for (int j = 0; j < 4; j += 2) {
            if (s == 1 && j == 0) continue;   // tokens 0 .. 15 see none of 16 .. 31
            uint32_t b[4];
            ldmatrix_x4(b[0], b[1], b[2], b[3], ab + j * 8 * LDA * 2 + s * 32);
            mma_bf16_16816(o[j], vf, b[0], b[1]);
            mma_bf16_16816(o[j + 1], vf, b[2], b[3]);
          }
#pragma unroll
          for (int k = 0; k < KT; ++k) {
            if (k >= cl.kt) break;
            uint32_t b[4];
            ldmatrix_x4_trans(b[0], b[1], b[2], b[3], kb + s * 16 * ldq * 2 + k * 32);
            mma_bf16_16816(S[2 * k], vf, b[0], b[1]);
            mma_bf16_16816(S[2 * k + 1], vf, b[2], b[3]);
          }
        }
        scale_state(f + Kp);
        if constexpr (CLUSTER) {
#pragma unroll
          for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[j][e] += o2[j][e];
        }
        // output and its sums of squares over this warp's value rows
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            const int t = j * 8 + 2 * t4 + e;
            float ss = o[j][e] * o[j][e] + o[j][e + 2] * o[j][e + 2];
            ss += __shfl_xor_sync(0xffffffffu, ss, 4);
            ss += __shfl_xor_sync(0xffffffffu, ss, 8);
            ss += __shfl_xor_sync(0xffffffffu, ss, 16);
            if (g == 0) ss_buf[warp * C + t] = ss;
            o_buf[t * ldO + warp * 16 + g] = o[j][e];
            o_buf[t * ldO + warp * 16 + g + 8] = o[j][e + 2];
          }
      }
    } else {
      // ---- token by token
      const bf16* sV = reinterpret_cast<const bf16*>(blk + cl.v);
      for (int t = 0; t < nt; ++t) {
        for (int k = tid; k < Kp; k += nthreads) {
          float q = 0.f, kk = 0.f, al = 0.f;
          if (k < K) {
            const float* x = base + t * ld;
            float z = m.a2_b[h * K + k];
            for (int s = 0; s < a.nsplit; ++s, x += a.split_stride) {
              q += x[h * K + k];
              kk += x[HK + h * K + k];
              for (int r = 0; r < m.rank; ++r) z = fmaf(x[2 * HK + 2 * HV + r], m.a2[r * HK + h * K + k], z);
            }
            al = ex2(-neg_log2_sigmoid(z) / m.tau);
          }
          sX[k] = q * rsqrtf((float)K);
          sX[Kp + k] = kk;
          sX[2 * Kp + k] = al;
        }
        __syncthreads();
        {
          const float va = __bfloat162float(sV[t * ldv + v0 + warp * 16 + g]), vb = __bfloat162float(sV[t * ldv + v0 + warp * 16 + g + 8]);
          float oa = 0.f, ob = 0.f;
#pragma unroll
          for (int j = 0; j < 2 * KT; ++j) {
            if (j >= 2 * cl.kt) break;
            const float2 q = *reinterpret_cast<const float2*>(sX + j * 8 + 2 * t4), k = *reinterpret_cast<const float2*>(sX + Kp + j * 8 + 2 * t4),
                         al = *reinterpret_cast<const float2*>(sX + 2 * Kp + j * 8 + 2 * t4);
            S[j][0] = fmaf(al.x, S[j][0], k.x * va);
            S[j][1] = fmaf(al.y, S[j][1], k.y * va);
            S[j][2] = fmaf(al.x, S[j][2], k.x * vb);
            S[j][3] = fmaf(al.y, S[j][3], k.y * vb);
            oa = fmaf(q.x, S[j][0], fmaf(q.y, S[j][1], oa));
            ob = fmaf(q.x, S[j][2], fmaf(q.y, S[j][3], ob));
          }
          oa += __shfl_xor_sync(0xffffffffu, oa, 1);
          oa += __shfl_xor_sync(0xffffffffu, oa, 2);
          ob += __shfl_xor_sync(0xffffffffu, ob, 1);
          ob += __shfl_xor_sync(0xffffffffu, ob, 2);
          float ss = oa * oa + ob * ob;
          ss += __shfl_xor_sync(0xffffffffu, ss, 4);
          ss += __shfl_xor_sync(0xffffffffu, ss, 8);
          ss += __shfl_xor_sync(0xffffffffu, ss, 16);
          if (t4 == 0) {
            o_buf[t * ldO + warp * 16 + g] = oa;
            o_buf[t * ldO + warp * 16 + g + 8] = ob;
          }
          if (lane == 0) ss_buf[warp * C + t] = ss;
        }
        __syncthreads();
      }
    }
    __syncthreads();   // the block has been read, the output stands in o_buf
    if (tid == 0 && it + 2 < chunks) load(it + 2);
    // ---- norm over the head, gate, store
    float* const norms = sS + 2 * C;
    auto warps_sum = [&]() -> float {
      float x[8];
#pragma unroll
      for (int w = 0; w < 8; ++w) x[w] = w * 16 < vs ? ss_buf[w * C + tid] : 0.f;
      return ((x[0] + x[1]) + (x[2] + x[3])) + ((x[4] + x[5]) + (x[6] + x[7]));
    };
    if constexpr (CLUSTER) {
      if (tid < C) sS[(it & 1) * C + tid] = warps_sum();
      cg::this_cluster().sync();
      if (tid < C) {
        float x[4];
#pragma unroll
        for (unsigned r = 0; r < 4; ++r) x[r] = r < gridDim.x ? cg::this_cluster().map_shared_rank(sS, r)[(it & 1) * C + tid] : 0.f;
        norms[tid] = rsqrtf(fmaf((x[0] + x[1]) + (x[2] + x[3]), inv_v, a.eps));
      }
    } else {
      if (tid < C) norms[tid] = rsqrtf(fmaf(warps_sum(), inv_v, a.eps));
    }
    __syncthreads();
    if (writes) {
      const float4 w = *reinterpret_cast<const float4*>(m.norm + v0 + vc);
      bf16* op = reinterpret_cast<bf16*>(a.out) + (int64_t)(p.row0 + it * C + vt) * a.ldo + h * V + v0 + vc;
      auto silu = [](float z) { return __fdividef(z, 1.0f + ex2(-LOG2E * z)); };
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = vt + i * vstep;
        if (t >= nt) break;
        const float f = norms[t];
        const float4 x = *reinterpret_cast<const float4*>(o_buf + t * ldO + vc);
        *reinterpret_cast<uint2*>(op + i * vstep * ldo) = make_uint2(pack_bf16(x.x * f * w.x * silu(gz[i].x), x.y * f * w.y * silu(gz[i].y)),
                                                                     pack_bf16(x.z * f * w.z * silu(gz[i].z), x.w * f * w.w * silu(gz[i].w)));
      }
    }
  }
  {
#pragma unroll
    for (int j = 0; j < 2 * KT; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int v = v0 + warp * 16 + g + 8 * (e >> 1), k = 8 * j + 2 * t4 + (e & 1);
        if (v < V && k < K) st[k * a.ldv + v] = S[j][e];
      }
  }
  if constexpr (CLUSTER) cg::this_cluster().sync();   // a peer may still read this CTA's sums
}

}  // namespace

bool gla_chunk_ok(const GlaDims& m) { return m.dim % 8 == 0 && m.vdim % 8 == 0 && m.dim <= 128 && m.vdim <= 128 && m.rank <= 64; }
int gla_chunks(int n) { return (n + C - 1) / C; }
int2 gla_chunk_rows(const GlaPortion& p, int i) { return make_int2(p.row0 + i * C, std::min(C, p.n - i * C)); }
size_t gla_chunk_bytes(const GlaDims& m) { return (size_t)m.heads * layout_of(m).bytes; }

int gla_chunk_launch(Ctx* c, const GlaArgs& a) {
  if (a.count == 0) return REWB200_OK;
  RB_REQUIRE(gla_chunk_ok(a.m) && a.dtype == REWB200_BF16 && a.list && a.chunks && a.work, "gated linear attention: sizes without a chunk kernel");
  const ChunkLayout cl = layout_of(a.m);
  const int prep_smem = cl.bytes + (C * ((a.m.rank + 3) / 4 * 4) + C / 8 * 4) * 4;
  RB_CUDA(cudaFuncSetAttribute(gla_prepare_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, prep_smem));
  RB_CUDA(launch_k(gla_prepare_kernel, dim3((unsigned)a.m.heads, (unsigned)a.n_chunks), dim3(NT), prep_smem, c->stream, c->use_pdl, a, cl));
  ++g_launch_total;
  // few portions: a cluster of CTAs shares a head's value columns
  int nv = 1;
  while (nv < 4 && cl.vp % (nv * 2 * 16) == 0 && (int64_t)nv * a.m.heads * a.count < c->sm_count) nv *= 2;
  const int vs = cl.vp / nv, smem = 2 * cl.bytes + (2 * C * (vs + 4) + 3 * C + 2 * 8 * C + 3 * cl.kt * 16) * 4 + 16;
  const dim3 grid((unsigned)nv, (unsigned)a.m.heads, (unsigned)a.count);
  auto go = [&](auto kernel, bool cluster) -> int {
    RB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    RB_CUDA(cluster ? launch_k_cluster(kernel, grid, dim3(2 * vs), smem, c->stream, c->use_pdl, dim3(nv), a, cl, vs)
                    : launch_k(kernel, grid, dim3(2 * vs), smem, c->stream, c->use_pdl, a, cl, vs));
    ++g_launch_total;
    return REWB200_OK;
  };
  if (cl.kt <= 4) return nv > 1 ? go(gla_scan_kernel<4, true>, true) : go(gla_scan_kernel<4, false>, false);
  return nv > 1 ? go(gla_scan_kernel<8, true>, true) : go(gla_scan_kernel<8, false>, false);
}

}  // namespace rewb
