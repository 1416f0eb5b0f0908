// Gated delta rule of large prompt portions, in chunks of 32 tokens on the tensor cores.
//
// With b_t the running sum of the log decays of a head inside the chunk, S the state ahead of it, and
//   L_ts = beta_t e^(b_t - b_s) k_t . k_s  (s < t)      A_ts = e^(b_t - b_s) q_t . k_s  (s <= t)
// the corrections u of the chunk solve a triangular system, (I + L) U = diag(beta) (V - diag(e^b) K S), so with T = (I + L)^-1
//   W = T diag(beta e^b) K        U = T diag(beta) V - W S
//   o_t = e^(b_t) q_t S + sum_s A_ts u_s                S <- e^(b_end) (S) + sum_s e^(b_end - b_s) k_s u_s^T
// (the inverse of I + L as in the chunked form of delta rules: forward substitution).  Every exponent is <= 0.  Two launches:
//   delta_prepare_kernel   one CTA per chunk and head: unit queries and keys, decays, T (forward substitution on the two
//                          diagonal halves, products for the block below), W, T diag(beta) V, A, as one block in the layout
//                          the second kernel has in shared memory (one bulk store)
//   delta_scan_kernel      one CTA walks the chunks of a portion for one head (or for a slice of its value columns; a cluster
//                          shares the head): blocks arrive by bulk copies two chunks ahead, the state stays in registers.
//                          Warp w holds the transposed state [16 value rows][dim], whose accumulator fragments are also the
//                          A operand of S W^T and S q^T; U^T comes out in the layout of the next products' A operand.
// Norms, decays, the triangular inverse and the state are f32; operands of products are bf16 (the state and T as a high part
// and a remainder) and sums f32.
#include <cooperative_groups.h>

#include <algorithm>

#include "act.cuh"
#include "delta.cuh"
#include "ptx.cuh"

namespace cg = cooperative_groups;

namespace rewb {

extern int64_t g_launch_total;

namespace {

constexpr int C = 32;             // tokens of a chunk
constexpr int NT = 256;
constexpr float UNIT_EPS = 1e-6f;
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ void ldmatrix_x2(uint32_t& r0, uint32_t& r1, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r0), "=r"(r1) : "r"(addr));
}
// x, y = hi + lo, packed bf16 pairs
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(x, y);
  const __nv_bfloat162 h = *reinterpret_cast<const __nv_bfloat162*>(&hi);
  lo = pack_bf16(x - __low2float(h), y - __high2float(h));
}
__device__ __forceinline__ float2 unpack2(uint32_t v) {
  const __nv_bfloat162 h = *reinterpret_cast<const __nv_bfloat162*>(&v);
  return make_float2(__low2float(h), __high2float(h));
}
__device__ __forceinline__ void bulk_store_1d(void* dst, const void* src, uint32_t bytes) {
  asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(dst), "r"(smem_u32(src)), "r"(bytes) : "memory");
  asm volatile("cp.async.bulk.commit_group;" ::: "memory");
}
// the source of this thread's bulk stores may be overwritten (or cease to exist) afterwards
__device__ __forceinline__ void bulk_store_wait() { asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory"); }

// The block of one chunk and head (byte offsets), rows padded by 16 bytes so that ldmatrix meets no bank conflicts.
struct ChunkLayout {
  int kt;           // 16-channel steps of a key: dim padded to 16 kt
  int vp;           // value columns, padded to a multiple of 16
  int ldq, ldv;     // elements of a key and of a value row
  int w, k, v, a;   // e^b q [C][ldq] at 0, W [C][ldq], e^(b_end - b) k [C][ldq], T diag(beta) V [C][ldv], A [C][C + 8]
  int f;            // decay of the whole chunk
  int bytes;
};
constexpr int LDA = C + 8, LDL = C + 4;

__host__ ChunkLayout layout_of(const DeltaDims& m) {
  ChunkLayout c;
  c.kt = (m.dim + 15) / 16;
  c.vp = (m.vdim + 15) / 16 * 16;
  c.ldq = c.kt * 16 + 8;
  c.ldv = c.vp + 8;
  c.w = C * c.ldq * 2;
  c.k = 2 * c.w;
  c.v = 3 * c.w;
  c.a = c.v + C * c.ldv * 2;
  c.f = c.a + C * LDA * 2;
  c.bytes = (c.f + 16 + 127) / 128 * 128;
  return c;
}
// scratch of the first kernel behind the block: L, T [C][LDL] f32, the product below the diagonal [16][17], four bf16 forms of
// T [C][LDA], per token b, beta, e^b [C] each
constexpr int PREP_SCRATCH = (2 * C * LDL + 16 * 17 + 3 * C) * 4 + 4 * C * LDA * 2;

// grid (heads, chunks)
__global__ void __launch_bounds__(NT, 3) delta_prepare_kernel(DeltaArgs a, ChunkLayout cl) {
  extern __shared__ __align__(128) uint8_t smem[];
  const DeltaDims& m = a.m;
  const int K = m.dim, V = m.vdim, ldq = cl.ldq, ldv = cl.ldv;
  bf16* sQ = reinterpret_cast<bf16*>(smem);            // q, then e^b q
  bf16* sW = reinterpret_cast<bf16*>(smem + cl.w);     // k, then W
  bf16* sKe = reinterpret_cast<bf16*>(smem + cl.k);
  bf16* sV = reinterpret_cast<bf16*>(smem + cl.v);     // v, then T diag(beta) v
  bf16* sA = reinterpret_cast<bf16*>(smem + cl.a);
  float* sL = reinterpret_cast<float*>(smem + cl.bytes);
  float* sT = sL + C * LDL;
  float* sP = sT + C * LDL;
  float *sB = sP + 16 * 17, *sBeta = sB + C, *sE = sBeta + C;
  bf16* sTw = reinterpret_cast<bf16*>(sE + C);         // T diag(beta e^b): high part, remainder; T diag(beta): the same
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l8 = lane & 7, lq = lane >> 3, g = lane >> 2, t4 = lane & 3;
  const int h = blockIdx.x, hk = h / (m.heads / m.kv_heads);
  pdl_launch_dependents();
  pdl_wait();
  const int2 ch = a.chunks[blockIdx.y];                // first row, tokens
  const int nt = ch.y;
  // ---- rows: a warp has four, a lane four channels of each at a time (dim and vdim up to 128, multiples of 8)
  float4 q[4], k[4];
  {
    const bool on = lane * 4 < K, vis = lane * 4 < V;
    const bf16* base = reinterpret_cast<const bf16*>(a.x) + (int64_t)ch.x * a.ldx;
    uint2 rq[4], rk[4], rv[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int t = warp * 4 + u;
      const bf16* p = base + t * a.ldx;
      rq[u] = rk[u] = rv[u] = make_uint2(0u, 0u);
      if (t < nt && on) {
        rq[u] = *reinterpret_cast<const uint2*>(p + hk * K + lane * 4);
        rk[u] = *reinterpret_cast<const uint2*>(p + (m.kv_heads + hk) * K + lane * 4);
      }
      if (t < nt && vis) rv[u] = *reinterpret_cast<const uint2*>(p + 2 * m.kv_heads * K + h * V + lane * 4);
    }
    if (warp == 0) {
      // step sizes and decays, a token a lane
      float beta = 0.f, lg = 0.f;
      if (lane < nt) {
        const float* p = a.partial + (int64_t)(ch.x + lane) * a.ld + (int64_t)m.heads * V + h;
        float zb = 0.f, za = 0.f;
        for (int s = 0; s < a.nsplit; ++s) {
          zb += p[s * a.split_stride];
          za += p[s * a.split_stride + m.heads];
        }
        beta = sigmoid_act(zb);
        lg = -m.rate[h] * softplus_act(za + m.dt_bias[h]);
      }
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float x = __shfl_up_sync(0xffffffffu, lg, o);
        if (lane >= o) lg += x;
      }
      sB[lane] = lg;
      sBeta[lane] = beta;
      sE[lane] = expf(lg);
      if (lane == 31) *reinterpret_cast<float*>(smem + cl.f) = expf(lg);
    }
    const float qscale = rsqrtf((float)K);
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int t = warp * 4 + u;
      const float2 q0 = unpack2(rq[u].x), q1 = unpack2(rq[u].y), k0 = unpack2(rk[u].x), k1 = unpack2(rk[u].y);
      const float fq = qscale / sqrtf(warp_sum(q0.x * q0.x + q0.y * q0.y + q1.x * q1.x + q1.y * q1.y) + UNIT_EPS);
      const float fk = 1.0f / sqrtf(warp_sum(k0.x * k0.x + k0.y * k0.y + k1.x * k1.x + k1.y * k1.y) + UNIT_EPS);
      q[u] = make_float4(q0.x * fq, q0.y * fq, q1.x * fq, q1.y * fq);
      k[u] = make_float4(k0.x * fk, k0.y * fk, k1.x * fk, k1.y * fk);
      if (lane * 4 < cl.kt * 16) {
        *reinterpret_cast<uint2*>(sQ + t * ldq + lane * 4) = make_uint2(pack_bf16(q[u].x, q[u].y), pack_bf16(q[u].z, q[u].w));
        *reinterpret_cast<uint2*>(sW + t * ldq + lane * 4) = make_uint2(pack_bf16(k[u].x, k[u].y), pack_bf16(k[u].z, k[u].w));
      }
      if (lane * 4 < cl.vp) *reinterpret_cast<uint2*>(sV + t * ldv + lane * 4) = rv[u];
    }
  }
  __syncthreads();
  // ---- L and A: six 16 x 8 tiles on and below the diagonal of each
  for (int tile = warp; tile < 12; tile += 8) {
    const int which = tile / 6, i = tile % 6, mt = i < 2 ? 0 : 1, nn = i < 2 ? i : i - 2;   // which: 0 L, 1 A
    float s[4] = {0.f, 0.f, 0.f, 0.f};
    const uint32_t qa = smem_u32(which ? sQ : sW) + ((mt * 16 + (lq & 1) * 8 + l8) * ldq + (lq >> 1) * 8) * 2;
    const uint32_t ka = smem_u32(sW) + ((nn * 8 + l8) * ldq + (lq & 1) * 8) * 2;
#pragma unroll 4
    for (int x = 0; x < cl.kt; ++x) {
      uint32_t f[4], b0, b1;
      ldmatrix_x4(f[0], f[1], f[2], f[3], qa + x * 32);
      ldmatrix_x2(b0, b1, ka + x * 32);
      mma_bf16_16816(s, f, b0, b1);
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int t = mt * 16 + g + 8 * r, sc = nn * 8 + 2 * t4;
      const float bt = sB[t], d0 = expf(fminf(bt - sB[sc], 0.f)), d1 = expf(fminf(bt - sB[sc + 1], 0.f));
      if (which) {
        *reinterpret_cast<uint32_t*>(sA + t * LDA + sc) = pack_bf16(sc <= t ? s[2 * r] * d0 : 0.f, sc + 1 <= t ? s[2 * r + 1] * d1 : 0.f);
      } else {
        const float be = sBeta[t];
        sL[t * LDL + sc] = sc < t ? be * d0 * s[2 * r] : 0.f;
        sL[t * LDL + sc + 1] = sc + 1 < t ? be * d1 * s[2 * r + 1] : 0.f;
      }
    }
  }
  __syncthreads();
  // ---- e^b q and e^(b_end - b) k; T of the diagonal halves: a column a lane, forward substitution
#pragma unroll
  for (int u = 0; u < 4; ++u) {
    const int t = warp * 4 + u;
    const float e = sE[t], d = expf(fminf(sB[C - 1] - sB[t], 0.f));
    if (lane * 4 < cl.kt * 16) {
      *reinterpret_cast<uint2*>(sQ + t * ldq + lane * 4) = make_uint2(pack_bf16(q[u].x * e, q[u].y * e), pack_bf16(q[u].z * e, q[u].w * e));
      *reinterpret_cast<uint2*>(sKe + t * ldq + lane * 4) = make_uint2(pack_bf16(k[u].x * d, k[u].y * d), pack_bf16(k[u].z * d, k[u].w * d));
    }
  }
  if (warp < 2 && lane < 16) {
    const int o = warp * 16;
    float x[16];
#pragma unroll
    for (int t = 0; t < 16; ++t) {
      float v = t == lane ? 1.f : 0.f;
#pragma unroll
      for (int s = 0; s < t; ++s) v = fmaf(-sL[(o + t) * LDL + o + s], x[s], v);
      x[t] = v;
      sT[(o + t) * LDL + o + lane] = v;
    }
  }
  __syncthreads();
  {
    // below the diagonal: -T22 L21 T11
    const int i = tid >> 4, j = tid & 15;
    float p = 0.f;
#pragma unroll
    for (int s = 0; s < 16; ++s) p = fmaf(sL[(16 + i) * LDL + s], sT[s * LDL + j], p);
    sP[i * 17 + j] = p;
    __syncthreads();
    p = 0.f;
#pragma unroll
    for (int s = 0; s < 16; ++s) p = fmaf(sT[(16 + i) * LDL + 16 + s], sP[s * 17 + j], p);
    sT[(16 + i) * LDL + j] = -p;
    sT[i * LDL + 16 + j] = 0.f;
  }
  __syncthreads();
  for (int i = tid; i < C * C / 2; i += NT) {
    const int t = i / (C / 2), s = (i % (C / 2)) * 2;
    const float x = sT[t * LDL + s] * sBeta[s], y = sT[t * LDL + s + 1] * sBeta[s + 1];
    uint32_t hi, lo;
    split2(x * sE[s], y * sE[s + 1], hi, lo);
    *reinterpret_cast<uint32_t*>(sTw + t * LDA + s) = hi;
    *reinterpret_cast<uint32_t*>(sTw + (C + t) * LDA + s) = lo;
    split2(x, y, hi, lo);
    *reinterpret_cast<uint32_t*>(sTw + (2 * C + t) * LDA + s) = hi;
    *reinterpret_cast<uint32_t*>(sTw + (3 * C + t) * LDA + s) = lo;
  }
  __syncthreads();
  // ---- W and T diag(beta) V: a warp has 16 columns at a time, which nobody else reads
  for (int n = warp; n < cl.kt + cl.vp / 16; n += 8) {
    const bool val = n >= cl.kt;
    const int col = (val ? n - cl.kt : n) * 16, ld = val ? ldv : ldq;
    bf16* const d = val ? sV : sW;
    const uint32_t ta = smem_u32(sTw + (val ? 2 * C * LDA : 0)) + (((lq & 1) * 8 + l8) * LDA + (lq >> 1) * 8) * 2;
    float o[2][2][4];
#pragma unroll
    for (int e = 0; e < 16; ++e) o[e >> 3][(e >> 2) & 1][e & 3] = 0.f;
    uint32_t b[2][4];
#pragma unroll
    for (int s = 0; s < 2; ++s)
      ldmatrix_x4_trans(b[s][0], b[s][1], b[s][2], b[s][3], smem_u32(d) + ((s * 16 + (lq & 1) * 8 + l8) * ld + col + (lq >> 1) * 8) * 2);
#pragma unroll
    for (int mt = 0; mt < 2; ++mt)
#pragma unroll
      for (int s = 0; s <= mt; ++s)
#pragma unroll
        for (int part = 0; part < 2; ++part) {
          uint32_t f[4];
          ldmatrix_x4(f[0], f[1], f[2], f[3], ta + (part * C + mt * 16) * LDA * 2 + s * 32);
          mma_bf16_16816(o[mt][0], f, b[s][0], b[s][1]);
          mma_bf16_16816(o[mt][1], f, b[s][2], b[s][3]);
        }
    __syncwarp();
#pragma unroll
    for (int mt = 0; mt < 2; ++mt)
#pragma unroll
      for (int half = 0; half < 2; ++half)
#pragma unroll
        for (int r = 0; r < 2; ++r)
          *reinterpret_cast<uint32_t*>(d + (mt * 16 + g + 8 * r) * ld + col + half * 8 + 2 * t4) = pack_bf16(o[mt][half][2 * r], o[mt][half][2 * r + 1]);
  }
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
__global__ void __launch_bounds__(CLUSTER ? NT / 2 : NT, CLUSTER ? 3 : 2) delta_scan_kernel(DeltaArgs a, ChunkLayout cl, int vs) {
  extern __shared__ __align__(128) uint8_t smem[];
  const DeltaDims& m = a.m;
  const int K = m.dim, V = m.vdim, ldq = cl.ldq, ldv = cl.ldv, ldO = vs + 4, ld = (int)a.ld;
  float* sO = reinterpret_cast<float*>(smem + 2 * cl.bytes);                 // [2][C][ldO]
  float* sS = sO + 2 * C * ldO;                                              // [2][C] sums of squares, [C] norms, [2][8 warps][C] sums of squares
  uint64_t* full = reinterpret_cast<uint64_t*>(sS + 3 * C + 2 * 8 * C);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l8 = lane & 7, lq = lane >> 3, g = lane >> 2, t4 = lane & 3;
  const int h = blockIdx.y, v0 = blockIdx.x * vs;
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
    const float* const base = a.partial + (int64_t)(p.row0 + it * C) * a.ld + h * V + v0 + vc;
    float* const o_buf = sO + (it & 1) * C * ldO;
    float* const ss_buf = sS + 3 * C + (it & 1) * 8 * C;
    // the gates of the chunk are requested ahead of its products
    float4 gz[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      gz[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (writes && vt + i * vstep < nt) gz[i] = *reinterpret_cast<const float4*>(base + (vt + i * vstep) * ld);
    }
    for (int s = 1; s < a.nsplit; ++s)
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (writes && vt + i * vstep < nt) {
          const float4 w = *reinterpret_cast<const float4*>(base + s * a.split_stride + (vt + i * vstep) * ld);
          gz[i].x += w.x; gz[i].y += w.y; gz[i].z += w.z; gz[i].w += w.w;
        }
    if (ok) ok = mbar_wait(full + (it & 1), (it >> 1) & 1, a.status);
    {
      const uint32_t aQ = smem_u32(blk), aW = aQ + cl.w, aK = aQ + cl.k, aV = aQ + cl.v, aA = aQ + cl.a;
      const float f = *reinterpret_cast<const float*>(blk + cl.f);
      // the state as every earlier token left it: o^T [16 value rows][C] = S^T (e^b q)^T and w^T = S^T W^T
      float o[4][4], u[4][4];
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[j][e] = u[j][e] = 0.f;
      const uint32_t qb = aQ + (((lq >> 1) * 8 + l8) * ldq + (lq & 1) * 8) * 2, half = 16 * ldq * 2, toW = aW - aQ;
#pragma unroll
      for (int k = 0; k < KT; ++k) {
        if (k >= cl.kt) break;
        uint32_t sh[4], sl[4];
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          split2(S[2 * k][2 * r], S[2 * k][2 * r + 1], sh[r], sl[r]);
          split2(S[2 * k + 1][2 * r], S[2 * k + 1][2 * r + 1], sh[2 + r], sl[2 + r]);
        }
#pragma unroll
        for (int x = 0; x < 2; ++x) {
          uint32_t b[4], c[4];
          ldmatrix_x4(b[0], b[1], b[2], b[3], qb + toW + x * half + k * 32);
          ldmatrix_x4(c[0], c[1], c[2], c[3], qb + x * half + k * 32);
          mma_bf16_16816(u[2 * x], sh, b[0], b[1]);
          mma_bf16_16816(u[2 * x + 1], sh, b[2], b[3]);
          mma_bf16_16816(o[2 * x], sh, c[0], c[1]);
          mma_bf16_16816(o[2 * x + 1], sh, c[2], c[3]);
          mma_bf16_16816(u[2 * x], sl, b[0], b[1]);
          mma_bf16_16816(u[2 * x + 1], sl, b[2], b[3]);
          mma_bf16_16816(o[2 * x], sl, c[0], c[1]);
          mma_bf16_16816(o[2 * x + 1], sl, c[2], c[3]);
        }
      }
      // the corrections U^T, as the A operand of what follows
      uint32_t uf[2][4];
#pragma unroll
      for (int s = 0; s < 2; ++s) {
        uint32_t vf[4];   // value rows 0-7 and 8-15 of tokens 0-7 of the half, then of tokens 8-15
        ldmatrix_x4_trans(vf[0], vf[1], vf[2], vf[3], aV + ((s * 16 + (lq >> 1) * 8 + l8) * ldv + v0 + warp * 16 + (lq & 1) * 8) * 2);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 v = unpack2(vf[e]);
          const float* x = u[2 * s + (e >> 1)] + 2 * (e & 1);
          uf[s][e] = pack_bf16(v.x - x[0], v.y - x[1]);
        }
      }
      // o^T += U^T A^T, S^T = decay S^T + U^T k
      const uint32_t ab = aA + (((lq >> 1) * 8 + l8) * LDA + (lq & 1) * 8) * 2;
      const uint32_t kb = aK + (((lq & 1) * 8 + l8) * ldq + (lq >> 1) * 8) * 2;
#pragma unroll
      for (int j = 0; j < 2 * KT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[j][e] *= f;
#pragma unroll
      for (int s = 0; s < 2; ++s) {
#pragma unroll
        for (int j = 0; j < 4; j += 2) {
          if (s == 1 && j == 0) continue;   // tokens 0 .. 15 see none of 16 .. 31
          uint32_t b[4];
          ldmatrix_x4(b[0], b[1], b[2], b[3], ab + j * 8 * LDA * 2 + s * 32);
          mma_bf16_16816(o[j], uf[s], b[0], b[1]);
          mma_bf16_16816(o[j + 1], uf[s], b[2], b[3]);
        }
#pragma unroll
        for (int k = 0; k < KT; ++k) {
          if (k >= cl.kt) break;
          uint32_t b[4];
          ldmatrix_x4_trans(b[0], b[1], b[2], b[3], kb + s * half + k * 32);
          mma_bf16_16816(S[2 * k], uf[s], b[0], b[1]);
          mma_bf16_16816(S[2 * k + 1], uf[s], b[2], b[3]);
        }
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
        norms[tid] = m.scale / sqrtf(fmaf((x[0] + x[1]) + (x[2] + x[3]), inv_v, a.eps));
      }
    } else {
      if (tid < C) norms[tid] = m.scale / sqrtf(fmaf(warps_sum(), inv_v, a.eps));
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
#pragma unroll
  for (int j = 0; j < 2 * KT; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int v = v0 + warp * 16 + g + 8 * (e >> 1), k = 8 * j + 2 * t4 + (e & 1);
      if (v < V && k < K) st[k * a.ldv + v] = S[j][e];
    }
  if constexpr (CLUSTER) cg::this_cluster().sync();   // a peer may still read this CTA's sums
}

}  // namespace

bool delta_chunk_ok(const DeltaDims& m) { return m.dim % 8 == 0 && m.vdim % 8 == 0 && m.dim <= 128 && m.vdim <= 128; }
int delta_chunks(int n) { return (n + C - 1) / C; }
int2 delta_chunk_rows(const GlaPortion& p, int i) { return make_int2(p.row0 + i * C, std::min(C, p.n - i * C)); }
size_t delta_chunk_bytes(const DeltaDims& m) { return (size_t)m.heads * layout_of(m).bytes; }

int delta_chunk_launch(Ctx* c, const DeltaArgs& a) {
  if (a.count == 0) return REWB200_OK;
  RB_REQUIRE(delta_chunk_ok(a.m) && a.dtype == REWB200_BF16 && a.list && a.chunks && a.work, "delta rule: sizes without a chunk kernel");
  const ChunkLayout cl = layout_of(a.m);
  const int prep_smem = cl.bytes + PREP_SCRATCH;
  RB_CUDA(cudaFuncSetAttribute(delta_prepare_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, prep_smem));
  RB_CUDA(launch_k(delta_prepare_kernel, dim3((unsigned)a.m.heads, (unsigned)a.n_chunks), dim3(NT), prep_smem, c->stream, c->use_pdl, a, cl));
  ++g_launch_total;
  // few portions: a cluster of CTAs shares a head's value columns
  int nv = 1;
  while (nv < 4 && cl.vp % (nv * 2 * 16) == 0 && (int64_t)nv * a.m.heads * a.count < c->sm_count) nv *= 2;
  const int vs = cl.vp / nv, smem = 2 * cl.bytes + (2 * C * (vs + 4) + 3 * C + 2 * 8 * C) * 4 + 16;
  const dim3 grid((unsigned)nv, (unsigned)a.m.heads, (unsigned)a.count);
  auto go = [&](auto kernel, bool cluster) -> int {
    RB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    RB_CUDA(cluster ? launch_k_cluster(kernel, grid, dim3(2 * vs), smem, c->stream, c->use_pdl, dim3(nv), a, cl, vs)
                    : launch_k(kernel, grid, dim3(2 * vs), smem, c->stream, c->use_pdl, a, cl, vs));
    ++g_launch_total;
    return REWB200_OK;
  };
  if (cl.kt <= 4) return nv > 1 ? go(delta_scan_kernel<4, true>, true) : go(delta_scan_kernel<4, false>, false);
  return nv > 1 ? go(delta_scan_kernel<8, true>, true) : go(delta_scan_kernel<8, false>, false);
}

}  // namespace rewb
