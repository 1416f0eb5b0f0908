// Gated linear attention, token by token (see gla.cuh).  Projections arrive as f32 slabs; decays, state, output norm and
// gate are f32.
#include <math.h>

#include <algorithm>

#include "gla.cuh"
#include "ptx.cuh"

namespace rewb {

extern int64_t g_launch_total;

namespace {

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

// What a token brings to one head, in shared memory: (alpha, k, scaled q) per key channel, v, gate, the features of the
// decay projection, and partial outputs.
struct TokenSmem {
  float4* akq;
  float *v, *g, *a1, *o;
};
__device__ __forceinline__ TokenSmem carve(float* sm, const GlaDims& m, int ldv) {
  TokenSmem s;
  s.akq = reinterpret_cast<float4*>(sm);
  s.v = sm + 4 * m.dim;
  s.g = s.v + ldv;
  s.a1 = s.g + ldv;
  s.o = s.a1 + (m.rank + 3) / 4 * 4;   // every part starts on 16 bytes: ldv is a multiple of 4
  return s;
}
int token_floats(const GlaDims& m, int ldv) { return 4 * m.dim + 2 * ldv + (m.rank + 3) / 4 * 4; }

template <int NT>
__device__ __forceinline__ void load_token(const GlaArgs& a, const TokenSmem& s, int h, int64_t row) {
  const GlaDims& m = a.m;
  const int K = m.dim, V = m.vdim, tid = threadIdx.x;
  const int64_t HK = (int64_t)m.heads * K, HV = (int64_t)m.heads * V;
  const float* p = a.partial + row * a.ld;
  // the decay features feed the longest chain, so they are requested first
  for (int i = tid; i < m.rank; i += NT) s.a1[i] = slab_sum(a, p + 2 * HK + 2 * HV + i);
  const float* pk = p + (int64_t)h * K;
  const float* pv = p + 2 * HK + (int64_t)h * V;
  for (int i = tid; i < max(K, V); i += NT) {
    float q = 0.f, k = 0.f, v = 0.f, g = 0.f;
    const bool ik = i < K, iv = i < V;
#pragma unroll 4
    for (int n = 0; n < a.nsplit; ++n) {
      const int64_t at = n * a.split_stride + i;
      if (ik) q += pk[at], k += pk[HK + at];
      if (iv) v += pv[at], g += pv[HV + at];
    }
    if (ik) s.akq[i] = make_float4(0.f, k, q * rsqrtf((float)K), 0.f);
    if (iv) s.v[i] = v, s.g[i] = g;
  }
  __syncthreads();
  const float inv_tau = 1.0f / m.tau;
  for (int i = tid; i < K; i += NT) {
    const float* w = m.a2 + (int64_t)h * K + i;
    float z = m.a2_b[(int64_t)h * K + i];
#pragma unroll 8
    for (int r = 0; r < m.rank; ++r) z = fmaf(s.a1[r], w[r * HK], z);
    s.akq[i].x = expf(log_decay(z, inv_tau));
  }
  __syncthreads();
}

// Sums the `slices` partial outputs of the head, then norm, gate and store.  Ends with a barrier.
template <typename T, int NT>
__device__ __forceinline__ void finish_token(const GlaArgs& a, const TokenSmem& s, int slices, float* red, int h, int64_t row) {
  const int V = a.m.vdim, tid = threadIdx.x;
  float ss = 0.f;
  for (int i = tid; i < V; i += NT) {
    float o = 0.f;
    for (int u = 0; u < slices; ++u) o += s.o[u * a.ldv + i];
    s.o[i] = o;
    ss += o * o;
  }
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int w = 0; w < NT / 32; ++w) ss += red[w];
  const float f = 1.0f / sqrtf(ss / (float)V + a.eps);
  T* op = reinterpret_cast<T*>(a.out) + row * a.ldo + (int64_t)h * V;
  for (int i = tid; i < V; i += NT) {   // the thread's own sums
    const float g = s.g[i];
    op[i] = stf<T>(s.o[i] * f * a.m.norm[i] * (g / (1.0f + expf(-g))));
  }
  __syncthreads();
}

__device__ __forceinline__ GlaPortion portion_of(const GlaArgs& a, int i) {
  if (a.list) return a.list[i];
  return GlaPortion{i, 1, a.pos0[a.b0 + i], a.b0 + i, 0};
}

// grid (heads, portions).  The head's state stays in registers over the portion: a thread owns four neighbouring value
// columns of up to KI key channels, `slices` apart.
template <typename T, int NT, int KI>
__global__ void __launch_bounds__(NT, NT == 128 ? (KI <= 16 ? 4 : 3) : KI <= 8 ? 2 : 1) gla_recurrent_kernel(GlaArgs a, int slices) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[NT / 32];
  pdl_launch_dependents();
  const GlaDims& m = a.m;
  const int h = blockIdx.x, K = m.dim, V = m.vdim, vq = a.ldv / 4;
  // weights depend on no earlier kernel
  for (int r = threadIdx.x / 8; r < m.rank; r += NT / 8)
    for (int i = (threadIdx.x % 8) * 32; i < K; i += 256) prefetch_l2(m.a2 + ((int64_t)r * m.heads + h) * K + i);
  prefetch_floats(m.a2_b + (int64_t)h * K, K);
  prefetch_floats(m.norm, V);
  if (!a.early) pdl_wait();
  const GlaPortion p = portion_of(a, blockIdx.y);
  const TokenSmem s = carve(sm, m, a.ldv);
  const int sl = threadIdx.x / vq, c = threadIdx.x - sl * vq;
  const int nk = sl < slices ? (K - sl + slices - 1) / slices : 0;   // channels of this thread
  const int step = slices * a.ldv;
  float* st = a.state + ((int64_t)p.lane * m.heads + h) * K * a.ldv + sl * a.ldv + c * 4;
  float4 S[KI];
  const int held = p.pos0 > 0 ? nk : 0;   // a sequence starts from a state of zero
#pragma unroll
  for (int i = 0; i < KI; ++i) S[i] = i < held ? *reinterpret_cast<const float4*>(st + i * step) : make_float4(0.f, 0.f, 0.f, 0.f);
  if (a.early) pdl_wait();
  if (threadIdx.x < (unsigned)(a.ldv - V)) s.v[V + threadIdx.x] = 0.f;
  for (int t = 0; t < p.n; ++t) {
    load_token<NT>(a, s, h, p.row0 + t);
    if (nk > 0) {
      const float4 v = *reinterpret_cast<const float4*>(s.v + c * 4);
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
      const float4* akq = s.akq + sl;
#pragma unroll
      for (int i = 0; i < KI; ++i) {
        if (i < nk) {
          const float4 x = akq[i * slices];
          S[i].x = fmaf(x.x, S[i].x, x.y * v.x);
          S[i].y = fmaf(x.x, S[i].y, x.y * v.y);
          S[i].z = fmaf(x.x, S[i].z, x.y * v.z);
          S[i].w = fmaf(x.x, S[i].w, x.y * v.w);
          o.x = fmaf(x.z, S[i].x, o.x);
          o.y = fmaf(x.z, S[i].y, o.y);
          o.z = fmaf(x.z, S[i].z, o.z);
          o.w = fmaf(x.z, S[i].w, o.w);
        }
      }
      *reinterpret_cast<float4*>(s.o + sl * a.ldv + c * 4) = o;
    }
    if (t + 1 == p.n) {
      // addresses are computed afresh: kept from the loads they would cost two registers each
      float* to = st;
      int by = step;
      asm volatile("" : "+l"(to), "+r"(by));
#pragma unroll
      for (int i = 0; i < KI; ++i)
        if (i < nk) *reinterpret_cast<float4*>(to + i * by) = S[i];
    }
    __syncthreads();
    finish_token<T, NT>(a, s, slices, red, h, p.row0 + t);
  }
}

// The same with the state in global memory: any size.
template <typename T, int NT>
__global__ void __launch_bounds__(NT) gla_plain_kernel(GlaArgs a) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[NT / 32];
  pdl_launch_dependents();
  pdl_wait();
  const GlaDims& m = a.m;
  const int h = blockIdx.x, K = m.dim, V = m.vdim;
  const GlaPortion p = portion_of(a, blockIdx.y);
  const TokenSmem s = carve(sm, m, a.ldv);
  float* st = a.state + ((int64_t)p.lane * m.heads + h) * K * a.ldv;
  for (int t = 0; t < p.n; ++t) {
    load_token<NT>(a, s, h, p.row0 + t);
    const bool fresh = p.pos0 + t == 0;
    for (int i = threadIdx.x; i < V; i += NT) {
      float o = 0.f;
      for (int k = 0; k < K; ++k) {
        const float4 x = s.akq[k];
        float& S = st[(int64_t)k * a.ldv + i];
        S = fmaf(x.x, fresh ? 0.f : S, x.y * s.v[i]);
        o = fmaf(x.z, S, o);
      }
      s.o[i] = o;
    }
    __syncthreads();
    finish_token<T, NT>(a, s, 1, red, h, p.row0 + t);
  }
}

}  // namespace

int64_t gla_state_ld(int vdim) { return (vdim + 3) / 4 * 4; }

int gla_recurrent_launch(Ctx* c, const GlaArgs& a) {
  if (a.count == 0) return REWB200_OK;
  const dim3 grid((unsigned)a.m.heads, (unsigned)a.count);
  const bool bf = a.dtype == REWB200_BF16;
  auto go = [&](auto kernel, int nt, int slices, auto... extra) -> int {
    const size_t smem = (size_t)(token_floats(a.m, a.ldv) + slices * a.ldv) * sizeof(float);
    if (smem > 48 * 1024) RB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    RB_CUDA(launch_k(kernel, grid, dim3(nt), smem, c->stream, c->use_pdl, a, extra...));
    ++g_launch_total;
    return REWB200_OK;
  };
  const int vq = a.ldv / 4;
  auto slices_of = [&](int nt) { return std::min(nt / vq, a.m.dim); };
  auto ki_of = [&](int nt) { return slices_of(nt) > 0 ? (a.m.dim + slices_of(nt) - 1) / slices_of(nt) : 1 << 20; };
#define RB_GLA(NT, KI)                                                                            \
  (bf ? go(gla_recurrent_kernel<bf16, NT, KI>, NT, slices_of(NT), slices_of(NT))                  \
      : go(gla_recurrent_kernel<float, NT, KI>, NT, slices_of(NT), slices_of(NT)))
  if (c->gla_impl != 1) {
    // few heads and sequences: more threads on each, for latency
    if ((int64_t)a.m.heads * a.count <= 2 * c->sm_count && ki_of(512) <= 8) return RB_GLA(512, 8);
    if (ki_of(128) <= 8) return RB_GLA(128, 8);
    if (ki_of(128) <= 16) return RB_GLA(128, 16);
    if (ki_of(128) <= 32) return RB_GLA(128, 32);
    if (ki_of(512) <= 16) return RB_GLA(512, 16);
  }
#undef RB_GLA
  return bf ? go(gla_plain_kernel<bf16, 256>, 256, 1) : go(gla_plain_kernel<float, 256>, 256, 1);
}

}  // namespace rewb
