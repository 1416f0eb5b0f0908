// Kernels of lru.cuh; everything but the operands u and the stored output is f32.
#include <algorithm>

#include "act.cuh"
#include "lru.cuh"
#include "ptx.cuh"

namespace rewb {

extern int64_t g_launch_total;

namespace {


__device__ __forceinline__ GlaPortion portion_of(const LruArgs& a, int i) {
  if (a.list) return a.list[i];
  return GlaPortion{i, 1, a.pos0[a.b0 + i], a.b0 + i, 0};
}

// A lane owns one channel, TT tokens at a time.  NW == 1: grid (channels / 128, portions), a warp walks its portion.  NW > 1: grid (channels / 32,
// portions), the warps of a CTA take consecutive runs of TT tokens; each reduces its run to (decay, contribution), the runs'
// effects meet in shared memory, and every warp replays its run from the state it then knows.
template <typename T, int NW, int TT>
__global__ void __launch_bounds__(NW == 1 ? 128 : 32 * NW) lru_kernel(LruArgs a) {
  __shared__ float2 runs[2][NW][32];
  pdl_launch_dependents();
  const LruDims& m = a.m;
  const int warp = threadIdx.x >> 5, ln = threadIdx.x & 31, w = NW == 1 ? 0 : warp, width = m.blocks * m.n;
  const int ch = (NW == 1 ? blockIdx.x * 4 + warp : blockIdx.x) * 32 + ln;
  const bool on = ch < width;
  const int b = on ? ch / m.n : 0, j = ch - b * m.n;
  const float decay = on ? m.decay[ch] : 0.f, yb = on ? m.y_bias[ch] : 0.f;
  if (!a.early) pdl_wait();
  const GlaPortion p = portion_of(a, blockIdx.y);
  float* const st = a.state + (int64_t)p.lane * width + ch;
  float S = p.pos0 > 0 && on ? *st : 0.f;   // a sequence starts from a state of zero
  if (a.early) pdl_wait();
  const float* gp = a.gates + ((int64_t)b * a.rows + p.row0) * 2 * m.ldn + j;
  const T* up = reinterpret_cast<const T*>(a.u) + ((int64_t)b * a.rows + p.row0) * m.ldn + j;
  const float* yp = a.partial + (int64_t)p.row0 * a.ld + ch;
  T* op = reinterpret_cast<T*>(a.out) + (int64_t)p.row0 * a.ldo + ch;
  for (int t0 = 0, it = 0; t0 < p.n; t0 += NW * TT, ++it) {
    const int tb = t0 + w * TT, nt = on ? min(p.n - tb, TT) : 0;
    float r[TT], i[TT], u[TT], y[TT];
#pragma unroll
    for (int k = 0; k < TT; ++k) {
      r[k] = i[k] = u[k] = y[k] = 0.f;
      if (k >= nt) continue;
      const int64_t t = tb + k;
      r[k] = gp[t * 2 * m.ldn];
      i[k] = gp[t * 2 * m.ldn + m.ldn];
      u[k] = ldf<T>(up[t * m.ldn]);
      y[k] = yp[t * a.ld];
    }
    for (int s = 1; s < a.nsplit; ++s)
#pragma unroll
      for (int k = 0; k < TT; ++k)
        if (k < nt) y[k] += yp[s * a.split_stride + (tb + k) * a.ld];
    // r, i become the decay and the contribution of a token; tokens past the end change nothing
#pragma unroll
    for (int k = 0; k < TT; ++k) {
      if (k >= nt) {
        r[k] = 1.f;
        i[k] = 0.f;
        continue;
      }
      if constexpr (sizeof(T) == 2) {
        const float la = decay * sigmoid_fast(r[k]);
        r[k] = __expf(la);
        i[k] = sqrt_fast(one_minus_exp(2.0f * la, r[k] * r[k])) * sigmoid_fast(i[k]) * u[k];
      } else {
        const float la = decay * sigmoid_act(r[k]);
        i[k] = sqrtf(-expm1f(2.0f * la)) * sigmoid_act(i[k]) * u[k];
        r[k] = expf(la);
      }
    }
    float c = S;
    if constexpr (NW > 1) {
      float A = 1.f, B = 0.f;
#pragma unroll
      for (int k = 0; k < TT; ++k) {
        A *= r[k];
        B = fmaf(r[k], B, i[k]);
      }
      runs[it & 1][w][ln] = make_float2(A, B);
      __syncthreads();
#pragma unroll
      for (int v = 0; v < NW; ++v) {
        const float2 e = runs[it & 1][v][ln];
        if (v == w) c = S;
        S = fmaf(e.x, S, e.y);
      }
    }
#pragma unroll
    for (int k = 0; k < TT; ++k) {
      c = fmaf(r[k], c, i[k]);
      if (k < nt) op[(int64_t)(tb + k) * a.ldo] = stf<T>(c * (sizeof(T) == 2 ? gelu_tanh_fast(y[k] + yb) : gelu_tanh_act(y[k] + yb)) * m.scale);
    }
    if constexpr (NW == 1) S = c;
  }
  if (on && w == 0) *st = S;
}

__global__ void lru_decay_kernel(float* lam, int64_t n) {
  const int64_t i = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
  if (i < n) lam[i] = -8.0f * softplus_act(lam[i]);
}

}  // namespace

int lru_launch(Ctx* c, const LruArgs& a) {
  if (a.count == 0) return REWB200_OK;
  const int width = a.m.blocks * a.m.n;
  const bool bf = a.dtype == REWB200_BF16, wide = a.list && a.longest > 16, single = !a.list || a.longest == 1;
  const dim3 grid((unsigned)(wide ? (width + 31) / 32 : (width + 127) / 128), (unsigned)a.count), block(wide ? 256 : 128);
  auto go = [&](auto kernel) { return launch_k(kernel, grid, block, 0, c->stream, c->use_pdl, a); };
  RB_CUDA(wide ? (bf ? go(lru_kernel<bf16, 8, 8>) : go(lru_kernel<float, 8, 8>))
          : single ? (bf ? go(lru_kernel<bf16, 1, 1>) : go(lru_kernel<float, 1, 1>))
                   : (bf ? go(lru_kernel<bf16, 1, 8>) : go(lru_kernel<float, 1, 8>)));
  ++g_launch_total;
  return REWB200_OK;
}

int lru_decay_launch(Ctx* c, float* lam, int64_t n) {
  lru_decay_kernel<<<(unsigned)((n + 255) / 256), 256, 0, c->stream>>>(lam, n);
  RB_CUDA(cudaGetLastError());
  ++g_launch_total;
  return REWB200_OK;
}

}  // namespace rewb
