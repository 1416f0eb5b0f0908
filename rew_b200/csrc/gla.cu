// Gated linear attention, token by token (see gla.cuh).  Projections arrive as f32 slabs; decays, state, output norm and
// gate are f32.
#include <math.h>

#include <algorithm>

#include "gla.cuh"
#include "ptx.cuh"

namespace rewb {

extern int64_t g_launch_total;

namespace {

constexpr int NT = 512;
constexpr int MAX_SLICES = 64;   // key slices of a CTA

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
// ln(sigmoid(z)) / tau
__device__ __forceinline__ float log_decay(float z, float inv_tau) { return -(fmaxf(-z, 0.f) + log1pf(expf(-fabsf(z)))) * inv_tau; }

// A column of a row summed over the slabs, in slab order.
__device__ __forceinline__ float slab_sum(const GlaArgs& a, const float* p) {
  float v = 0.f;
#pragma unroll 4
  for (int s = 0; s < a.nsplit; ++s) v += p[s * a.split_stride];
  return v;
}

// What a token brings to one head, in shared memory: q (scaled), k, alpha [dim]; v, gate [vdim]; the decay projection's
// features.
struct TokenSmem {
  float *q, *k, *al, *v, *g, *a1;
};
__device__ __forceinline__ TokenSmem carve(float* sm, const GlaDims& m) {
  TokenSmem s;
  s.q = sm;
  s.k = s.q + m.dim;
  s.al = s.k + m.dim;
  s.v = s.al + m.dim;
  s.g = s.v + (m.vdim + 3) / 4 * 4;
  s.a1 = s.g + m.vdim;
  return s;
}
__device__ __forceinline__ void load_token(const GlaArgs& a, const TokenSmem& s, int h, int64_t row) {
  const GlaDims& m = a.m;
  const float qscale = rsqrtf((float)m.dim), inv_tau = 1.0f / m.tau;
  const int K = m.dim, V = m.vdim;
  const int64_t HK = (int64_t)m.heads * K, HV = (int64_t)m.heads * V;
  const float* p = a.partial + row * a.ld;
  // the decay features feed a longer chain: the last warp loads them, q, k, v and the gate go to all threads
  if (threadIdx.x >= NT - 32)
    for (int i = threadIdx.x - (NT - 32); i < m.rank; i += 32) s.a1[i] = slab_sum(a, p + 2 * HK + 2 * HV + i);
  for (int i = threadIdx.x; i < 2 * K + 2 * V; i += NT) {
    const bool key = i < 2 * K;
    const int j = key ? i : i - 2 * K, n = key ? K : V, second = j >= n ? 1 : 0, at = j - second * n;
    const float v = slab_sum(a, p + (key ? 0 : 2 * HK) + second * (key ? HK : HV) + (int64_t)h * n + at);
    (key ? (second ? s.k : s.q) : (second ? s.g : s.v))[at] = key && !second ? v * qscale : v;
  }
  __syncthreads();
  for (int i = threadIdx.x; i < K; i += NT) {
    const float* w = m.a2 + (int64_t)h * K + i;
    float z = m.a2_b[(int64_t)h * K + i];
#pragma unroll 8
    for (int r = 0; r < m.rank; ++r) z = fmaf(s.a1[r], w[r * HK], z);
    s.al[i] = expf(log_decay(z, inv_tau));
  }
  __syncthreads();
}
// Norm, gate and store of the head's output o [vdim] (shared memory, complete).
template <typename T>
__device__ __forceinline__ void finish_token(const GlaArgs& a, const TokenSmem& s, const float* o, float* red, int h, int64_t row) {
  const int V = a.m.vdim;
  float ss = 0.f;
  for (int i = threadIdx.x; i < V; i += NT) ss += o[i] * o[i];
  ss = warp_sum(ss);
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int w = 0; w < NT / 32; ++w) ss += red[w];
  const float f = 1.0f / sqrtf(ss / (float)V + a.eps);
  T* op = reinterpret_cast<T*>(a.out) + row * a.ldo + (int64_t)h * V;
  for (int i = threadIdx.x; i < V; i += NT) {
    const float g = s.g[i];
    op[i] = stf<T>(o[i] * f * a.m.norm[i] * (g / (1.0f + expf(-g))));
  }
  __syncthreads();
}

__device__ __forceinline__ GlaPortion portion_of(const GlaArgs& a, int i) {
  if (a.list) return a.list[i];
  return GlaPortion{i, 1, a.pos0[a.b0 + i], a.b0 + i};
}

// grid (heads, portions).  The head's state stays in registers over the portion: a thread owns four neighbouring value
// columns of KI key channels.
template <typename T, int KI>
__global__ void __launch_bounds__(NT, KI <= 8 ? 2 : 1) gla_recurrent_kernel(GlaArgs a, int slices) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[NT / 32];
  pdl_launch_dependents();
  const GlaDims& m = a.m;
  const int h = blockIdx.x, K = m.dim, V = m.vdim, vq = a.ldv / 4;
  if (!a.early) pdl_wait();
  const GlaPortion p = portion_of(a, blockIdx.y);
  const TokenSmem s = carve(sm, m);
  float* so = s.a1 + (m.rank + 3) / 4 * 4;                    // [slices][ldv]
  so = reinterpret_cast<float*>((reinterpret_cast<uintptr_t>(so) + 15) & ~uintptr_t(15));
  const int c = threadIdx.x % vq, sl = threadIdx.x / vq;
  const bool on = sl < slices;
  float* st = a.state + ((int64_t)p.lane * m.heads + h) * K * a.ldv + c * 4;
  float4 S[KI];
#pragma unroll
  for (int i = 0; i < KI; ++i) {
    const int k = sl + i * slices;
    S[i] = on && k < K && p.pos0 > 0 ? *reinterpret_cast<const float4*>(st + (int64_t)k * a.ldv) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  if (a.early) pdl_wait();
  if (threadIdx.x >= (unsigned)V && threadIdx.x < (unsigned)a.ldv) s.v[threadIdx.x] = 0.f;
  for (int t = 0; t < p.n; ++t) {
    const int64_t row = p.row0 + t;
    load_token(a, s, h, row);
    if (on) {
      const float4 v = make_float4(s.v[c * 4], s.v[c * 4 + 1], s.v[c * 4 + 2], s.v[c * 4 + 3]);
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int i = 0; i < KI; ++i) {
        const int k = sl + i * slices;
        if (k < K) {
          const float al = s.al[k], kk = s.k[k], q = s.q[k];
          S[i].x = fmaf(al, S[i].x, kk * v.x);
          S[i].y = fmaf(al, S[i].y, kk * v.y);
          S[i].z = fmaf(al, S[i].z, kk * v.z);
          S[i].w = fmaf(al, S[i].w, kk * v.w);
          o.x = fmaf(q, S[i].x, o.x);
          o.y = fmaf(q, S[i].y, o.y);
          o.z = fmaf(q, S[i].z, o.z);
          o.w = fmaf(q, S[i].w, o.w);
        }
      }
      *reinterpret_cast<float4*>(so + sl * a.ldv + c * 4) = o;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < V; i += NT) {
      float v = 0.f;
      for (int u = 0; u < slices; ++u) v += so[u * a.ldv + i];
      so[i] = v;
    }
    __syncthreads();
    finish_token<T>(a, s, so, red, h, row);
  }
#pragma unroll
  for (int i = 0; i < KI; ++i) {
    const int k = sl + i * slices;
    if (on && k < K) *reinterpret_cast<float4*>(st + (int64_t)k * a.ldv) = S[i];
  }
}

// The same with the state in global memory: any size.
template <typename T>
__global__ void __launch_bounds__(NT) gla_plain_kernel(GlaArgs a) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[NT / 32];
  pdl_launch_dependents();
  pdl_wait();
  const GlaDims& m = a.m;
  const int h = blockIdx.x, K = m.dim, V = m.vdim;
  const GlaPortion p = portion_of(a, blockIdx.y);
  const TokenSmem s = carve(sm, m);
  float* so = s.a1 + m.rank;
  float* st = a.state + ((int64_t)p.lane * m.heads + h) * K * a.ldv;
  for (int t = 0; t < p.n; ++t) {
    const int64_t row = p.row0 + t;
    load_token(a, s, h, row);
    const bool fresh = p.pos0 + t == 0;
    for (int i = threadIdx.x; i < V; i += NT) {
      float o = 0.f;
      for (int k = 0; k < K; ++k) {
        float& S = st[(int64_t)k * a.ldv + i];
        S = fmaf(s.al[k], fresh ? 0.f : S, s.k[k] * s.v[i]);
        o = fmaf(s.q[k], S, o);
      }
      so[i] = o;
    }
    __syncthreads();
    finish_token<T>(a, s, so, red, h, row);
  }
}

}  // namespace

int64_t gla_state_ld(int vdim) { return (vdim + 3) / 4 * 4; }

int gla_recurrent_launch(Ctx* c, const GlaArgs& a) {
  if (a.count == 0) return REWB200_OK;
  const dim3 grid((unsigned)a.m.heads, (unsigned)a.count);
  const int vq = a.ldv / 4, slices = std::min({MAX_SLICES, NT / std::max(vq, 1), a.m.dim});
  const int ki = slices > 0 ? (a.m.dim + slices - 1) / slices : 1 << 20;
  const bool bf = a.dtype == REWB200_BF16;
  const int token = 3 * a.m.dim + 2 * a.ldv + a.m.rank + 8;
  auto go = [&](auto kernel, size_t smem, auto... extra) -> int {
    if (smem > 48 * 1024) RB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    RB_CUDA(launch_k(kernel, grid, dim3(NT), smem, c->stream, c->use_pdl, a, extra...));
    ++g_launch_total;
    return REWB200_OK;
  };
  if (c->gla_impl == 1 || ki > 16) {
    const size_t smem = (size_t)(token + a.ldv) * sizeof(float);
    return bf ? go(gla_plain_kernel<bf16>, smem) : go(gla_plain_kernel<float>, smem);
  }
  const size_t smem = (size_t)(token + slices * a.ldv + 8) * sizeof(float);
#define RB_GLA(KI) (bf ? go(gla_recurrent_kernel<bf16, KI>, smem, slices) : go(gla_recurrent_kernel<float, KI>, smem, slices))
  return ki <= 2 ? RB_GLA(2) : ki <= 4 ? RB_GLA(4) : ki <= 8 ? RB_GLA(8) : RB_GLA(16);
#undef RB_GLA
}

}  // namespace rewb
