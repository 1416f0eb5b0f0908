// Gated linear attention of large prompt portions, in chunks of 32 tokens on the tensor cores.
//
// With b_t the running sum of the log decays of a key channel and r its value in the middle of the chunk,
//   q~_t = q_t e^(b_t - r)      k~_s = k_s e^(r - b_s)      A_ts = q~_t . k~_s  (s <= t)
//   o_t  = q~_t (e^r S) + sum_s A_ts v_s                    S <- e^(b_end - r) (e^r S + sum_s k~_s v_s^T)
// so one pair of scaled operands serves the scores, the output and the state.  A CTA walks the chunks of one portion
// with the state of one head (or of a slice of its value columns; a cluster shares the head) in registers: warp w holds
// the transposed state [16 value rows][dim], whose accumulator fragments are also the A operand of q~ S.  Decays, their
// sums and the state are f32; operands of products are bf16 (the state as a high part and a remainder) and sums f32.
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
__device__ __forceinline__ void prefetch_l2(const void* p) { asm volatile("prefetch.global.L2 [%0];" ::"l"(p)); }
// x, y = hi + lo, packed bf16 pairs
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(x, y);
  const __nv_bfloat162 h = *reinterpret_cast<const __nv_bfloat162*>(&hi);
  lo = pack_bf16(x - __low2float(h), y - __high2float(h));
}
struct ChunkCfg {
  int kt;        // 16-channel steps of a key: dim padded to 16 kt
  int vs;        // value columns of the CTA, a multiple of 16
  int rp;        // decay features padded to a multiple of 4
  int ldq;       // elements of a row of the q~ / k~ buffers
  int off_k, off_v, off_a, off_a1, off_a2, off_f, off_ss;   // byte offsets in shared memory (q~ and the staged output at 0)
};

// KT: capacity of the register state in 16-channel steps.
template <int KT, bool CLUSTER>
__global__ void __launch_bounds__(NT, 2) gla_chunk_kernel(GlaArgs a, ChunkCfg cf) {
  extern __shared__ __align__(16) uint8_t smem[];
  const GlaDims& m = a.m;
  const int K = m.dim, V = m.vdim, Kp = cf.kt * 16, vs = cf.vs, rp = cf.rp, ldq = cf.ldq, ldv = vs + 8, ldO = vs + 4;
  bf16* sQ = reinterpret_cast<bf16*>(smem);                    // [C][ldq]
  float* sO = reinterpret_cast<float*>(smem);                  // [C][ldO], once q~ has been read
  bf16* sK = reinterpret_cast<bf16*>(smem + cf.off_k);         // [C][ldq]
  bf16* sV = reinterpret_cast<bf16*>(smem + cf.off_v);         // [C][ldv]
  bf16* sA = reinterpret_cast<bf16*>(smem + cf.off_a);         // [C][C + 8]
  float* sA1 = reinterpret_cast<float*>(smem + cf.off_a1);     // [2][a1_at(C, 0)]
  float* sA2 = reinterpret_cast<float*>(smem + cf.off_a2);     // [rp][Kp]
  float* sF = reinterpret_cast<float*>(smem + cf.off_f);       // [Kp] decay up to the middle since the state was scaled last
  float* sEnd = sF + Kp;                                       // [2][Kp] decay after the middle, by chunk parity
  float* sS = reinterpret_cast<float*>(smem + cf.off_ss);      // [2][C] sums of squares (cluster), then [8 warps][C]
  constexpr int ldA = C + 8;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l8 = lane & 7, lq = lane >> 3, g = lane >> 2, t4 = lane & 3;
  const int h = blockIdx.y, v0 = blockIdx.x * vs;
  const int HK = m.heads * K, HV = m.heads * V;
  const bool state_warp = warp * 16 < vs;
  pdl_launch_dependents();
  // weights of the decay projection do not depend on earlier kernels
  for (int i = tid; i < rp * Kp; i += NT) {
    const int r = i / Kp, k = i % Kp;
    sA2[i] = r < m.rank && k < K ? m.a2[r * HK + h * K + k] : 0.f;
  }
  // this thread's pair of key channels and eight tokens: a warp has 32 channels of one half of the chunk, its upper lanes
  // the later eight tokens
  const int half = warp >> 2, kc = (warp & 3) * 32 + (lane & 15) * 2, late = lane >> 4, tb = half * 16 + late * 8;
  const bool mine = kc < Kp, live = kc < K;
  const uint32_t pair = __ballot_sync(0xffffffffu, mine);      // both lanes of a channel pair are in or out together
  for (int k = tid; k < Kp; k += NT) sEnd[Kp + k] = 1.f;       // the chunk before the first one
  // rows of decay features, with a gap every eight of them so that two groups of lanes read different banks
  auto a1_at = [rp](int t, int r) { return t * rp + (t >> 3) * 4 + r; };
  const int a1_size = a1_at(C, 0), ld = (int)a.ld;
  pdl_wait();
  const GlaPortion p = a.list[blockIdx.z];
  auto state = [&]() -> float* { return a.state + ((int64_t)p.lane * m.heads + h) * K * a.ldv; };
  // S[j][e]: value row v0 + 16 warp + g + 8 (e >> 1), channel 8 j + 2 t4 + (e & 1)
  float S[2 * KT][4];
#pragma unroll
  for (int j = 0; j < 2 * KT; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int v = v0 + warp * 16 + g + 8 * (e >> 1), k = 8 * j + 2 * t4 + (e & 1);
      S[j][e] = p.pos0 > 0 && state_warp && v < V && k < K ? state()[k * a.ldv + v] : 0.f;
    }
  // items of four columns this thread handles of a [C][vs] tile: one column group, tokens vt, vt + vstep, ..
  const int vq = vs / 4, vt = tid / vq, vc = (tid % vq) * 4, vstep = NT / vq;   // vs <= 128: at most 4 items
  const bool exact = NT % vq == 0 && C % vstep == 0 && v0 + vs <= V;
  auto tile4 = [&](const float* base, int nt, float4 (&x)[4]) {
    const float* b = base + vt * ld + vc;
    if (exact && nt == C && a.nsplit == 1) {
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (i * vstep < C) x[i] = *reinterpret_cast<const float4*>(b + i * vstep * ld);
      return;
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      x[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (vt < vstep && vt + i * vstep < nt && v0 + vc < V)
        for (int s = 0; s < a.nsplit; ++s) {
          const float4 w = *reinterpret_cast<const float4*>(b + s * a.split_stride + i * vstep * ld);
          x[i].x += w.x; x[i].y += w.y; x[i].z += w.z; x[i].w += w.w;
        }
    }
  };
  auto load_a1 = [&](int t0, float* dst) {
    for (int i = tid; i < C * rp; i += NT) {
      const int t = i / rp, r = i % rp;
      float v = 0.f;
      if (t0 + t < p.n && r < m.rank) {
        const float* x = a.partial + (int64_t)(p.row0 + t0 + t) * a.ld + 2 * HK + 2 * HV + r;
        for (int s = 0; s < a.nsplit; ++s) v += x[s * a.split_stride];
      }
      dst[a1_at(t, r)] = v;
    }
  };
  load_a1(0, sA1);
  __syncthreads();
  const float qscale = rsqrtf((float)K), dscale = -1.0f / m.tau, inv_v = 1.0f / (float)V;
  for (int t0 = 0, it = 0; t0 < p.n; t0 += C, ++it) {
    const int nt = min(C, p.n - t0);
    const float* a1 = sA1 + (it & 1) * a1_size;
    float* const end_prev = sEnd + ((it & 1) ^ 1) * Kp;
    float* const end_now = sEnd + (it & 1) * Kp;
    const float* base = a.partial + (int64_t)(p.row0 + t0) * a.ld;
    // ---- values
    {
      float4 x[4];
      tile4(base + 2 * HK + h * V + v0, nt, x);
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = vt + i * vstep;
        if (vt < vstep && t < C) *reinterpret_cast<uint2*>(sV + t * ldv + vc) = make_uint2(pack_bf16(x[i].x, x[i].y), pack_bf16(x[i].z, x[i].w));
      }
    }
    // ---- decays and scaled queries and keys of this thread's channels and tokens
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
      float2 e[8];
      const float2 kbias = live ? *reinterpret_cast<const float2*>(m.a2_b + h * K + kc) : make_float2(0.f, 0.f);
#pragma unroll
      for (int u = 0; u < 8; ++u) e[u] = kbias;
      for (int r = 0; r < rp; r += 4) {
        float2 w[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) w[i] = *reinterpret_cast<const float2*>(sA2 + (r + i) * Kp + kc);
#pragma unroll
        for (int u = 0; u < 8; ++u) {
          const float4 x = *reinterpret_cast<const float4*>(a1 + a1_at(tb + u, r));
          e[u].x = fmaf(x.x, w[0].x, fmaf(x.y, w[1].x, fmaf(x.z, w[2].x, fmaf(x.w, w[3].x, e[u].x))));
          e[u].y = fmaf(x.x, w[0].y, fmaf(x.y, w[1].y, fmaf(x.z, w[2].y, fmaf(x.w, w[3].y, e[u].y))));
        }
      }
      // log2 of the decays, then their sums from the middle of the chunk
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
      if (!late) {
        const float2 f = make_float2(ex2(tot.x), ex2(tot.y));
        if (half) {
          *reinterpret_cast<float2*>(end_now + kc) = f;
        } else {
          const float2 g0 = *reinterpret_cast<const float2*>(end_prev + kc);
          *reinterpret_cast<float2*>(sF + kc) = make_float2(f.x * g0.x, f.y * g0.y);
        }
      }
      // first half: minus the decays still ahead of the middle; second half: the decays since
      float2 run = half ? (late ? other : make_float2(0.f, 0.f)) : (late ? part : tot);
      bf16* dq = sQ + tb * ldq + kc;
      bf16* dk = sK + tb * ldq + kc;
#pragma unroll
      for (int u = 0; u < 8; ++u) {
        if (half) {
          run.x += e[u].x;
          run.y += e[u].y;
          e[u] = run;
        } else {
          run.x -= e[u].x;
          run.y -= e[u].y;
          e[u] = make_float2(-run.x, -run.y);
        }
        if (far) e[u] = make_float2(0.f, 0.f);
      }
      float2 x[8];
      rows8(qp, x);
#pragma unroll
      for (int u = 0; u < 8; ++u)
        *reinterpret_cast<uint32_t*>(dq + u * ldq) = pack_bf16(x[u].x * (qscale * ex2(e[u].x)), x[u].y * (qscale * ex2(e[u].y)));
      rows8(qp + HK, x);
#pragma unroll
      for (int u = 0; u < 8; ++u) *reinterpret_cast<uint32_t*>(dk + u * ldq) = pack_bf16(x[u].x * ex2(-e[u].x), x[u].y * ex2(-e[u].y));
    }
    const bool slow = __syncthreads_or(far ? 1 : 0) != 0;
    if (t0 + C < p.n) {
      load_a1(t0 + C, sA1 + ((it + 1) & 1) * a1_size);
      // the next chunk's rows of this head move into L2 under this chunk's products
      const int line = (tid & 3) * 32, part = (tid >> 2) & 3;
      if (line < (part < 2 ? K : vs)) {
        const float* x = base + (C + (tid >> 4)) * ld + (part < 2 ? part * HK + h * K : 2 * HK + (part - 2) * HV + h * V + v0) + line;
        if (t0 + C + (tid >> 4) < p.n) prefetch_l2(x);
        if (t0 + C + 16 + (tid >> 4) < p.n) prefetch_l2(x + 16 * ld);
      }
    }
    float o[4][4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) o[j][e] = 0.f;
    if (!slow) {
      const uint32_t aQ = smem_u32(sQ), aK = smem_u32(sK), aV = smem_u32(sV), aA = smem_u32(sA);
      // ---- scores: six 16 x 8 tiles on and below the diagonal
      if (warp < 6) {
        const int mt = warp < 2 ? 0 : 1, nn = warp < 2 ? warp : warp - 2;
        float s[4] = {0.f, 0.f, 0.f, 0.f};
        const uint32_t qa = aQ + ((mt * 16 + (lq & 1) * 8 + l8) * ldq + (lq >> 1) * 8) * 2;
        const uint32_t ka = aK + ((nn * 8 + l8) * ldq + (lq & 1) * 8) * 2;
#pragma unroll
        for (int k = 0; k < KT; ++k) {
          if (k >= cf.kt) break;
          uint32_t q[4], b0, b1;
          ldmatrix_x4(q[0], q[1], q[2], q[3], qa + k * 32);
          ldmatrix_x2(b0, b1, ka + k * 32);
          mma_bf16_16816(s, q, b0, b1);
        }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          const int t = mt * 16 + g + 8 * r, sc = nn * 8 + 2 * t4;
          *reinterpret_cast<uint32_t*>(sA + t * ldA + sc) = pack_bf16(sc <= t ? s[2 * r] : 0.f, sc + 1 <= t ? s[2 * r + 1] : 0.f);
        }
      }
      // ---- the state as every earlier token left it: o^T [16 value rows][C] = (e^r S)^T q~^T
      if (state_warp) {
        const uint32_t qb = aQ + (((lq >> 1) * 8 + l8) * ldq + (lq & 1) * 8) * 2, qb2 = qb + 16 * ldq * 2;
#pragma unroll
        for (int k = 0; k < KT; ++k) {
          if (k >= cf.kt) break;
          const float2 f0 = *reinterpret_cast<const float2*>(sF + k * 16 + 2 * t4), f1 = *reinterpret_cast<const float2*>(sF + k * 16 + 8 + 2 * t4);
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
#pragma unroll
          for (int j = 0; j < 4; j += 2) {
            uint32_t b[4];
            ldmatrix_x4(b[0], b[1], b[2], b[3], (j ? qb2 : qb) + k * 32);
            mma_bf16_16816(o[j], sh, b[0], b[1]);
            mma_bf16_16816(o[j + 1], sh, b[2], b[3]);
            mma_bf16_16816(o[j], sl, b[0], b[1]);
            mma_bf16_16816(o[j + 1], sl, b[2], b[3]);
          }
        }
      }
      __syncthreads();
      // ---- o^T += v^T A^T, S^T += v^T k~; the decay after the middle joins the next scaling of the state
      if (state_warp) {
        const uint32_t ab = aA + (((lq >> 1) * 8 + l8) * ldA + (lq & 1) * 8) * 2;
        const uint32_t kb = aK + (((lq & 1) * 8 + l8) * ldq + (lq >> 1) * 8) * 2, kb2 = kb + 16 * ldq * 2;
#pragma unroll
        for (int s = 0; s < 2; ++s) {
          uint32_t vf[4];
          ldmatrix_x4_trans(vf[0], vf[1], vf[2], vf[3], aV + ((s * 16 + (lq >> 1) * 8 + l8) * ldv + warp * 16 + (lq & 1) * 8) * 2);
#pragma unroll
          for (int j = 0; j < 4; j += 2) {
            if (s == 1 && j == 0) continue;   // tokens 0 .. 15 see none of 16 .. 31
            uint32_t b[4];
            ldmatrix_x4(b[0], b[1], b[2], b[3], ab + j * 8 * ldA * 2 + s * 32);
            mma_bf16_16816(o[j], vf, b[0], b[1]);
            mma_bf16_16816(o[j + 1], vf, b[2], b[3]);
          }
#pragma unroll
          for (int k = 0; k < KT; ++k) {
            if (k >= cf.kt) break;
            uint32_t b[4];
            ldmatrix_x4_trans(b[0], b[1], b[2], b[3], (s ? kb2 : kb) + k * 32);
            mma_bf16_16816(S[2 * k], vf, b[0], b[1]);
            mma_bf16_16816(S[2 * k + 1], vf, b[2], b[3]);
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
            if (g == 0) sS[2 * C + warp * C + t] = ss;
            sO[t * ldO + warp * 16 + g] = o[j][e];
            sO[t * ldO + warp * 16 + g + 8] = o[j][e + 2];
          }
      }
    } else {
      // ---- token by token: q | k | alpha in the k~ buffer
      float* x = reinterpret_cast<float*>(sK);
#pragma unroll
      for (int j = 0; j < 2 * KT; ++j) {
        if (j >= 2 * cf.kt) break;
        const float2 f = *reinterpret_cast<const float2*>(end_prev + j * 8 + 2 * t4);
        S[j][0] *= f.x;
        S[j][1] *= f.y;
        S[j][2] *= f.x;
        S[j][3] *= f.y;
      }
      for (int k = tid; k < Kp; k += NT) end_now[k] = 1.f;
      for (int t = 0; t < nt; ++t) {
        for (int k = tid; k < Kp; k += NT) {
          float q = 0.f, kk = 0.f, al = 0.f;
          if (k < K) {
            const float* qp = base + t * ld + h * K + k;
            for (int s = 0; s < a.nsplit; ++s) {
              q += qp[s * a.split_stride];
              kk += qp[s * a.split_stride + HK];
            }
            q *= qscale;
            float z = m.a2_b[h * K + k];
            for (int r = 0; r < rp; ++r) z = fmaf(a1[a1_at(t, r)], sA2[r * Kp + k], z);
            al = ex2(neg_log2_sigmoid(z) * dscale);
          }
          x[k] = q;
          x[Kp + k] = kk;
          x[2 * Kp + k] = al;
        }
        __syncthreads();
        if (state_warp) {
          const float va = __bfloat162float(sV[t * ldv + warp * 16 + g]), vb = __bfloat162float(sV[t * ldv + warp * 16 + g + 8]);
          float oa = 0.f, ob = 0.f;
#pragma unroll
          for (int j = 0; j < 2 * KT; ++j) {
            if (j >= 2 * cf.kt) break;
            const float2 q = *reinterpret_cast<const float2*>(x + j * 8 + 2 * t4), k = *reinterpret_cast<const float2*>(x + Kp + j * 8 + 2 * t4),
                         al = *reinterpret_cast<const float2*>(x + 2 * Kp + j * 8 + 2 * t4);
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
            sO[t * ldO + warp * 16 + g] = oa;
            sO[t * ldO + warp * 16 + g + 8] = ob;
          }
          if (lane == 0) sS[2 * C + warp * C + t] = ss;
        }
        __syncthreads();
      }
    }
    // the gates are requested ahead of the barrier
    float4 gz[4];
    tile4(base + 2 * HK + HV + h * V + v0, nt, gz);
    __syncthreads();
    // ---- norm over the head, gate, store
    if (tid < C) {
      float ss = 0.f;
      for (int w = 0; w * 16 < vs; ++w) ss += sS[2 * C + w * C + tid];
      sS[(it & 1) * C + tid] = CLUSTER ? ss : rsqrtf(fmaf(ss, inv_v, a.eps));
    }
    if constexpr (CLUSTER) cg::this_cluster().sync();
    else __syncthreads();
    if (vt < vstep && v0 + vc < V) {
      const float4 w = *reinterpret_cast<const float4*>(m.norm + v0 + vc);
      bf16* op = reinterpret_cast<bf16*>(a.out) + (int64_t)(p.row0 + t0 + vt) * a.ldo + h * V + v0 + vc;
      const int ldo = (int)a.ldo;
      auto silu = [](float z) { return __fdividef(z, 1.0f + ex2(-LOG2E * z)); };
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = vt + i * vstep;
        if (t >= nt) break;
        float f = sS[(it & 1) * C + t];
        if constexpr (CLUSTER) {
          f = 0.f;
          for (unsigned r = 0; r < gridDim.x; ++r) f += cg::this_cluster().map_shared_rank(sS, r)[(it & 1) * C + t];
          f = rsqrtf(fmaf(f, inv_v, a.eps));
        }
        const float4 x = *reinterpret_cast<const float4*>(sO + t * ldO + vc);
        *reinterpret_cast<uint2*>(op + i * vstep * ldo) = make_uint2(pack_bf16(x.x * f * w.x * silu(gz[i].x), x.y * f * w.y * silu(gz[i].y)),
                                                                     pack_bf16(x.z * f * w.z * silu(gz[i].z), x.w * f * w.w * silu(gz[i].w)));
      }
    }
    __syncthreads();
  }
  if (state_warp) {
    const float* f = sEnd + (((p.n + C - 1) / C - 1) & 1) * Kp;
    float* to = state();
#pragma unroll
    for (int j = 0; j < 2 * KT; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int v = v0 + warp * 16 + g + 8 * (e >> 1), k = 8 * j + 2 * t4 + (e & 1);
        if (v < V && k < K) to[k * a.ldv + v] = S[j][e] * f[k];
      }
  }
  if constexpr (CLUSTER) cg::this_cluster().sync();   // a peer may still read this CTA's sums
}

}  // namespace

bool gla_chunk_ok(const GlaDims& m) { return m.dim % 8 == 0 && m.vdim % 8 == 0 && m.dim <= 128 && m.vdim <= 128 && m.rank <= 64; }

int gla_chunk_launch(Ctx* c, const GlaArgs& a) {
  if (a.count == 0) return REWB200_OK;
  RB_REQUIRE(gla_chunk_ok(a.m) && a.dtype == REWB200_BF16 && a.list, "gated linear attention: sizes without a chunk kernel");
  const int vp = (a.m.vdim + 15) / 16 * 16;
  // few portions: a cluster of CTAs shares a head's value columns
  int nv = 1;
  while (nv < 4 && vp % (nv * 2 * 16) == 0 && (int64_t)nv * a.m.heads * a.count < c->sm_count) nv *= 2;
  ChunkCfg cf;
  cf.kt = (a.m.dim + 15) / 16;
  cf.vs = vp / nv;
  cf.rp = (a.m.rank + 3) / 4 * 4;
  const int Kp = cf.kt * 16;
  cf.ldq = Kp + 8;
  auto up = [](int v) { return (v + 127) / 128 * 128; };
  const int ops = C * cf.ldq * 2;
  cf.off_k = up(std::max(ops, C * (cf.vs + 4) * 4));
  cf.off_v = cf.off_k + up(std::max(ops, 3 * Kp * 4));
  cf.off_a = cf.off_v + up(C * (cf.vs + 8) * 2);
  cf.off_a1 = cf.off_a + up(C * (C + 8) * 2);
  cf.off_a2 = cf.off_a1 + up(2 * (C * cf.rp + C / 8 * 4) * 4);
  cf.off_f = cf.off_a2 + up(cf.rp * Kp * 4);
  cf.off_ss = cf.off_f + up(3 * Kp * 4);
  const int smem = cf.off_ss + up((2 + 8) * C * 4);
  const dim3 grid((unsigned)nv, (unsigned)a.m.heads, (unsigned)a.count);
  auto go = [&](auto kernel, bool cluster) -> int {
    RB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    RB_CUDA(cluster ? launch_k_cluster(kernel, grid, dim3(NT), smem, c->stream, c->use_pdl, dim3(nv), a, cf)
                    : launch_k(kernel, grid, dim3(NT), smem, c->stream, c->use_pdl, a, cf));
    ++g_launch_total;
    return REWB200_OK;
  };
  if (cf.kt <= 4) return nv > 1 ? go(gla_chunk_kernel<4, true>, true) : go(gla_chunk_kernel<4, false>, false);
  return nv > 1 ? go(gla_chunk_kernel<8, true>, true) : go(gla_chunk_kernel<8, false>, false);
}

}  // namespace rewb
