// Gated delta rule, token by token (see delta.cuh).  Unit norms, decays, step sizes, state, output norm and gate are f32.
#include <algorithm>

#include "act.cuh"
#include "delta.cuh"
#include "ptx.cuh"

namespace rewb {

extern int64_t g_launch_total;

namespace {

constexpr float UNIT_EPS = 1e-6f;

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  return v;
}
__device__ __forceinline__ float slab_sum(const DeltaArgs& a, const float* p) {
  float v = 0.f;
#pragma unroll 4
  for (int s = 0; s < a.nsplit; ++s) v += p[s * a.split_stride];
  return v;
}

// What a token brings to one head, in shared memory: (k, q) per key channel as they leave the convolution, v, gate, and the
// partial sums over key channels of S^T k and S^T q.
struct TokenSmem {
  float2* kq;
  float *v, *g, *pk, *pq;
};
__device__ __forceinline__ TokenSmem carve(float* sm, int Kp, int ldv, int slices) {
  TokenSmem s;
  s.kq = reinterpret_cast<float2*>(sm);
  s.v = sm + 2 * Kp;
  s.g = s.v + ldv;
  s.pk = s.g + ldv;
  s.pq = s.pk + slices * ldv;
  return s;
}
int token_floats(int Kp, int ldv, int slices) { return 2 * Kp + 2 * ldv + 2 * slices * ldv; }

struct TokenScalars {
  float beta, g, rk, rq, kq;   // step size, decay, factors of the raw key and query, their product
};

// Loads a token; every thread returns its scalars.  Ends with a barrier.
template <typename T, int NT>
__device__ __forceinline__ TokenScalars load_token(const DeltaArgs& a, const TokenSmem& s, int h, int64_t row) {
  const DeltaDims& m = a.m;
  const int K = m.dim, V = m.vdim, tid = threadIdx.x, hk = h / (m.heads / m.kv_heads);
  const float* p = a.partial + row * a.ld;
  const float zb = slab_sum(a, p + (int64_t)m.heads * V + h), za = slab_sum(a, p + (int64_t)m.heads * V + m.heads + h);
  const T* x = reinterpret_cast<const T*>(a.x) + row * a.ldx;
  const T *q = x + (int64_t)hk * K, *k = q + (int64_t)m.kv_heads * K, *v = x + 2 * (int64_t)m.kv_heads * K + (int64_t)h * V;
  for (int i = tid; i < K; i += NT) s.kq[i] = make_float2(ldf<T>(k[i]), ldf<T>(q[i]));
  for (int i = tid; i < V; i += NT) {
    s.v[i] = ldf<T>(v[i]);
    s.g[i] = slab_sum(a, p + (int64_t)h * V + i);
  }
  __syncthreads();
  float kk = 0.f, qq = 0.f, kq = 0.f;
  for (int i = tid & 31; i < K; i += 32) {
    const float2 e = s.kq[i];
    kk = fmaf(e.x, e.x, kk);
    qq = fmaf(e.y, e.y, qq);
    kq = fmaf(e.x, e.y, kq);
  }
  kk = warp_sum(kk);
  qq = warp_sum(qq);
  kq = warp_sum(kq);
  TokenScalars t;
  t.rk = 1.0f / sqrtf(kk + UNIT_EPS);
  t.rq = 1.0f / (sqrtf(qq + UNIT_EPS) * sqrtf((float)K));
  t.kq = kq * t.rk * t.rq;
  t.beta = sigmoid_act(zb);
  t.g = expf(-m.rate[h] * softplus_act(za + m.dt_bias[h]));
  return t;
}

// Norm, gate and store of the head's output, which the NT threads hold `o` of: column `col` .. col + 3 of the threads with
// `mine`.  Ends with a barrier.
template <typename T, int NT>
__device__ __forceinline__ void finish_token(const DeltaArgs& a, const TokenSmem& s, float4 o, bool mine, int col, float* red, int h, int64_t row) {
  const int V = a.m.vdim, tid = threadIdx.x;
  float ss = mine ? o.x * o.x + o.y * o.y + o.z * o.z + o.w * o.w : 0.f;   // columns past V are zero
  ss = warp_sum(ss);
  if ((tid & 31) == 0) red[tid >> 5] = ss;
  __syncthreads();
  ss = 0.f;
#pragma unroll
  for (int w = 0; w < NT / 32; ++w) ss += red[w];
  const float f = a.m.scale / sqrtf(ss / (float)V + a.eps);
  if (mine) {
    T* op = reinterpret_cast<T*>(a.out) + row * a.ldo + (int64_t)h * V;
    const float e[4] = {o.x, o.y, o.z, o.w};
#pragma unroll
    for (int u = 0; u < 4; ++u)
      if (col + u < V) op[col + u] = stf<T>(e[u] * f * a.m.norm[col + u] * silu_act(s.g[col + u]));
  }
  __syncthreads();
}

__device__ __forceinline__ GlaPortion portion_of(const DeltaArgs& a, int i) {
  if (a.list) return a.list[i];
  return GlaPortion{i, 1, a.pos0[a.b0 + i], a.b0 + i, 0};
}

// grid (heads, portions).  The head's state stays in registers over the portion: a thread owns four neighbouring value
// columns of up to KI key channels, `slices` apart.  One pass over the state gives S^T k and S^T q:
//   u = beta (v - g S^T k),  o = g S^T q + (k . q) u,  S <- g S + k u^T
template <typename T, int NT, int KI>
__global__ void __launch_bounds__(NT, NT == 128 ? (KI <= 16 ? 4 : 3) : KI <= 8 ? 2 : 1) delta_recurrent_kernel(DeltaArgs a, int slices) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[NT / 32];
  pdl_launch_dependents();
  const DeltaDims& m = a.m;
  const int h = blockIdx.x, K = m.dim, V = m.vdim, vq = a.ldv / 4;
  prefetch_floats(m.norm, V);
  if (!a.early) pdl_wait();
  const GlaPortion p = portion_of(a, blockIdx.y);
  const TokenSmem s = carve(sm, (K + 1) / 2 * 2, a.ldv, slices);
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
    const TokenScalars x = load_token<T, NT>(a, s, h, p.row0 + t);
    const float2* kq = s.kq + sl;
    if (nk > 0) {
      float4 uk = make_float4(0.f, 0.f, 0.f, 0.f), uq = uk;
#pragma unroll
      for (int i = 0; i < KI; ++i) {
        if (i < nk) {
          const float2 e = kq[i * slices];
          uk.x = fmaf(e.x, S[i].x, uk.x);
          uk.y = fmaf(e.x, S[i].y, uk.y);
          uk.z = fmaf(e.x, S[i].z, uk.z);
          uk.w = fmaf(e.x, S[i].w, uk.w);
          uq.x = fmaf(e.y, S[i].x, uq.x);
          uq.y = fmaf(e.y, S[i].y, uq.y);
          uq.z = fmaf(e.y, S[i].z, uq.z);
          uq.w = fmaf(e.y, S[i].w, uq.w);
        }
      }
      *reinterpret_cast<float4*>(s.pk + sl * a.ldv + c * 4) = uk;
      *reinterpret_cast<float4*>(s.pq + sl * a.ldv + c * 4) = uq;
    }
    __syncthreads();
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
    if (nk > 0) {
      float4 uk = o, uq = o;
      for (int r = 0; r < slices; ++r) {
        const float4 e = *reinterpret_cast<const float4*>(s.pk + r * a.ldv + c * 4);
        uk.x += e.x; uk.y += e.y; uk.z += e.z; uk.w += e.w;
      }
      if (sl == 0)
        for (int r = 0; r < slices; ++r) {
          const float4 e = *reinterpret_cast<const float4*>(s.pq + r * a.ldv + c * 4);
          uq.x += e.x; uq.y += e.y; uq.z += e.z; uq.w += e.w;
        }
      const float4 v = *reinterpret_cast<const float4*>(s.v + c * 4);
      const float gk = x.g * x.rk, gq = x.g * x.rq;
      const float4 u = make_float4(x.beta * (v.x - gk * uk.x), x.beta * (v.y - gk * uk.y), x.beta * (v.z - gk * uk.z), x.beta * (v.w - gk * uk.w));
      o = make_float4(fmaf(gq, uq.x, x.kq * u.x), fmaf(gq, uq.y, x.kq * u.y), fmaf(gq, uq.z, x.kq * u.z), fmaf(gq, uq.w, x.kq * u.w));
#pragma unroll
      for (int i = 0; i < KI; ++i) {
        if (i < nk) {
          const float k = kq[i * slices].x * x.rk;
          S[i].x = fmaf(x.g, S[i].x, k * u.x);
          S[i].y = fmaf(x.g, S[i].y, k * u.y);
          S[i].z = fmaf(x.g, S[i].z, k * u.z);
          S[i].w = fmaf(x.g, S[i].w, k * u.w);
        }
      }
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
    finish_token<T, NT>(a, s, o, sl == 0, c * 4, red, h, p.row0 + t);
  }
}

// The same with the state in global memory: any size.  A thread owns four value columns at a time.
template <typename T, int NT>
__global__ void __launch_bounds__(NT) delta_plain_kernel(DeltaArgs a) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[NT / 32];
  pdl_launch_dependents();
  pdl_wait();
  const DeltaDims& m = a.m;
  const int h = blockIdx.x, K = m.dim, V = m.vdim;
  const GlaPortion p = portion_of(a, blockIdx.y);
  const TokenSmem s = carve(sm, (K + 1) / 2 * 2, a.ldv, 1);
  float* st = a.state + ((int64_t)p.lane * m.heads + h) * K * a.ldv;
  for (int t = 0; t < p.n; ++t) {
    const TokenScalars x = load_token<T, NT>(a, s, h, p.row0 + t);
    const bool fresh = p.pos0 + t == 0;
    float ss = 0.f;
    for (int i = threadIdx.x; i < V; i += NT) {
      float uk = 0.f, uq = 0.f;
      for (int k = 0; k < K && !fresh; ++k) {
        const float2 e = s.kq[k];
        const float S = st[(int64_t)k * a.ldv + i];
        uk = fmaf(e.x, S, uk);
        uq = fmaf(e.y, S, uq);
      }
      const float u = x.beta * (s.v[i] - x.g * x.rk * uk), o = fmaf(x.g * x.rq, uq, x.kq * u);
      for (int k = 0; k < K; ++k) {
        float& S = st[(int64_t)k * a.ldv + i];
        S = fmaf(x.g, fresh ? 0.f : S, s.kq[k].x * x.rk * u);
      }
      s.pq[i] = o;
      ss += o * o;
    }
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.f;
    for (int w = 0; w < NT / 32; ++w) ss += red[w];
    const float f = m.scale / sqrtf(ss / (float)V + a.eps);
    T* op = reinterpret_cast<T*>(a.out) + (int64_t)(p.row0 + t) * a.ldo + (int64_t)h * V;
    for (int i = threadIdx.x; i < V; i += NT) op[i] = stf<T>(s.pq[i] * f * m.norm[i] * silu_act(s.g[i]));   // the thread's own sums
    __syncthreads();
  }
}

__global__ void delta_rate_kernel(float* p, int64_t n) {
  const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) p[i] = expf(p[i]);
}

}  // namespace

int delta_rate_launch(Ctx* c, float* a_log, int64_t n) {
  delta_rate_kernel<<<(unsigned)((n + 255) / 256), 256, 0, c->stream>>>(a_log, n);
  RB_CUDA(cudaGetLastError());
  ++g_launch_total;
  return REWB200_OK;
}

int delta_recurrent_launch(Ctx* c, const DeltaArgs& a) {
  if (a.count == 0) return REWB200_OK;
  const dim3 grid((unsigned)a.m.heads, (unsigned)a.count);
  const bool bf = a.dtype == REWB200_BF16;
  const int Kp = (a.m.dim + 1) / 2 * 2;
  auto go = [&](auto kernel, int nt, int slices, auto... extra) -> int {
    const size_t smem = (size_t)token_floats(Kp, a.ldv, slices) * sizeof(float);
    if (smem > 48 * 1024) RB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    RB_CUDA(launch_k(kernel, grid, dim3(nt), smem, c->stream, c->use_pdl, a, extra...));
    ++g_launch_total;
    return REWB200_OK;
  };
  const int vq = a.ldv / 4;
  auto slices_of = [&](int nt) { return std::min(nt / vq, a.m.dim); };
  auto ki_of = [&](int nt) { return slices_of(nt) > 0 ? (a.m.dim + slices_of(nt) - 1) / slices_of(nt) : 1 << 20; };
#define RB_DELTA(NT, KI)                                                                          \
  (bf ? go(delta_recurrent_kernel<bf16, NT, KI>, NT, slices_of(NT), slices_of(NT))                \
      : go(delta_recurrent_kernel<float, NT, KI>, NT, slices_of(NT), slices_of(NT)))
  if (c->gla_impl != 1) {
    // few heads and sequences: more threads on each, for latency
    if ((int64_t)a.m.heads * a.count <= 2 * c->sm_count && ki_of(512) <= 8) return RB_DELTA(512, 8);
    if (ki_of(128) <= 8) return RB_DELTA(128, 8);
    if (ki_of(128) <= 16) return RB_DELTA(128, 16);
    if (ki_of(128) <= 32) return RB_DELTA(128, 32);
    if (ki_of(512) <= 16) return RB_DELTA(512, 16);
  }
#undef RB_DELTA
  return bf ? go(delta_plain_kernel<bf16, 256>, 256, 1) : go(delta_plain_kernel<float, 256>, 256, 1);
}

}  // namespace rewb
