// Kernels of gqa_mix.cuh for any dtype and size.  Scores, softmax, mixing and gates are f32.
#include <math.h>

#include <algorithm>

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

}  // namespace

size_t gqa_mix_bytes(Ctx* c, const GqaDims& m, int dtype, int64_t rows, int64_t tiles, int64_t max_tile_rows, int64_t max_ctx) {
  (void)c; (void)dtype; (void)tiles; (void)max_tile_rows;
  const size_t row = (size_t)m.heads * most_seen(m, max_ctx) * sizeof(float);
  return std::max(row, std::min(PLAIN_WORK, row * (size_t)rows));
}

int gqa_mix_launch(Ctx* c, const GqaMixArgs& a) {
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

}  // namespace rewb
