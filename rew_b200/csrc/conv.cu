// Kernels of conv.cuh.  Inputs, sums and state are f32.
#include <algorithm>

#include "act.cuh"
#include "conv.cuh"
#include "ptx.cuh"

namespace rewb {

extern int64_t g_launch_total;

namespace {

constexpr int NT = 128, MAX_TR = 32;

__device__ __forceinline__ void add4(float4& v, float4 w) { v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w; }
__device__ __forceinline__ void fma4(float4& y, float4 w, float4 x) {
  y.x = fmaf(w.x, x.x, y.x);
  y.y = fmaf(w.y, x.y, y.y);
  y.z = fmaf(w.z, x.z, y.z);
  y.w = fmaf(w.w, x.w, y.w);
}
// Rows of the same portion ahead of `row` in this step, at most `most`.
__device__ __forceinline__ int rows_ahead(const RowMap& m, int64_t row, int lane, int pos, int most) {
  int n = 0;
  if (m.row_lane)
    while (n < most && row - n - 1 >= 0 && m.row_lane[row - n - 1] == lane && m.row_pos[row - n - 1] == pos - n - 1) ++n;
  return n;
}

// grid (rows / tr, channels / 512): a thread owns four channels and walks down tr rows with the last TAPS - 1 inputs in
// registers.
template <typename T, int TAPS>
__global__ void __launch_bounds__(NT) conv_kernel(ConvArgs a, int64_t rows, int tr) {
  __shared__ int4 info[MAX_TR];   // per row: position (-1: outside the cache), lane, rows of its portion ahead of it
  pdl_launch_dependents();
  const int64_t row0 = (int64_t)blockIdx.x * tr, C = a.m.channels, ch = ((int64_t)blockIdx.y * NT + threadIdx.x) * 4;
  const int nr = (int)min((int64_t)tr, rows - row0);
  const bool on = ch < C;
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  float4 w[TAPS], bi = zero, bo = zero;   // weights by tokens ago
#pragma unroll
  for (int b = 0; b < TAPS; ++b) w[b] = on && b < a.m.taps ? *reinterpret_cast<const float4*>(a.m.w + (a.m.taps - 1 - b) * C + ch) : zero;
  if (on && a.m.in_bias) bi = *reinterpret_cast<const float4*>(a.m.in_bias + ch);
  if (on && a.m.bias) bo = *reinterpret_cast<const float4*>(a.m.bias + ch);
  if (!a.early) pdl_wait();
  if ((int)threadIdx.x < nr) {
    const int64_t row = row0 + threadIdx.x;
    const int lane = row_lane(a.map, row), pos = row_pos(a.map, row);
    const bool in = pos >= 0 && pos < a.capacity;
    if (!in && blockIdx.y == 0) atomicExch(a.status, KS_BAD_INDEX);
    info[threadIdx.x] = make_int4(in ? pos : -1, lane, rows_ahead(a.map, row, lane, pos, TAPS - 1), 0);
  }
  __syncthreads();
  const int slots = a.m.taps - 1;
  auto state_at = [&](int lane, int pos) { return reinterpret_cast<float4*>(a.state + ((int64_t)lane * slots + pos % slots) * C + ch); };
  float4 h[TAPS];     // inputs by tokens ago
#pragma unroll
  for (int b = 0; b < TAPS; ++b) h[b] = zero;
  auto from_state = [&](const int4& in, int first) {
#pragma unroll
    for (int b = 1; b < TAPS; ++b)
      if (b >= first && on && b < a.m.taps && in.x - b >= 0) h[b] = *state_at(in.y, in.x - b);
      else if (b >= first) h[b] = zero;
  };
  from_state(info[0], info[0].z + 1);
  if (a.early) pdl_wait();
  const float* p = a.partial + row0 * a.ld + ch;
  auto value = [&](const float* x) {
    float4 v = bi;
    if (!on) return zero;
#pragma unroll 4
    for (int s = 0; s < a.nsplit; ++s) add4(v, *reinterpret_cast<const float4*>(x + s * a.split_stride));
    return v;
  };
#pragma unroll
  for (int b = 1; b < TAPS; ++b)
    if (b <= info[0].z && b < a.m.taps) h[b] = value(p - b * a.ld);
  const int64_t g = a.group > 0 ? ch / a.group : 0;
  T* out = reinterpret_cast<T*>(a.out) + (a.group > 0 ? (g * rows + row0) * a.ldo + ch - g * a.group : row0 * a.ldo + ch);
  const bool keep = !a.tails && a.m.taps > 1 && on;
  constexpr int AHEAD = TAPS <= 4 ? 8 : 4;    // rows requested together
  for (int r0 = 0; r0 < nr; r0 += AHEAD) {
    float4 xs[AHEAD];
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) xs[u] = on && r0 + u < nr ? *reinterpret_cast<const float4*>(p + (r0 + u) * a.ld) : zero;
    for (int s = 1; s < a.nsplit; ++s)
#pragma unroll
      for (int u = 0; u < AHEAD; ++u)
        if (on && r0 + u < nr) add4(xs[u], *reinterpret_cast<const float4*>(p + s * a.split_stride + (r0 + u) * a.ld));
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) add4(xs[u], bi);
#pragma unroll
    for (int u = 0; u < AHEAD; ++u) {
      const int r = r0 + u;
      if (r >= nr) break;
      const int4 in = info[r];
      if (r > 0 && in.z == 0) from_state(in, 1);    // a portion starts here
      h[0] = xs[u];
      float4 y = bo;
#pragma unroll
      for (int b = 0; b < TAPS; ++b) fma4(y, w[b], h[b]);
      if (keep && in.x >= 0) *state_at(in.y, in.x) = h[0];
#pragma unroll
      for (int b = TAPS - 1; b > 0; --b) h[b] = h[b - 1];
      if (a.m.silu)
        y = sizeof(T) == 2 ? make_float4(silu_fast(y.x), silu_fast(y.y), silu_fast(y.z), silu_fast(y.w))
                           : make_float4(silu_act(y.x), silu_act(y.y), silu_act(y.z), silu_act(y.w));
      if (!on) continue;
      if constexpr (sizeof(T) == 2) *reinterpret_cast<uint2*>(out + r * a.ldo) = make_uint2(pack_bf16(y.x, y.y), pack_bf16(y.z, y.w));
      else *reinterpret_cast<float4*>(out + r * a.ldo) = y;
    }
  }
  if (a.offsets && a.group > 0 && blockIdx.x == 0 && blockIdx.y == 0)
    for (int64_t i = threadIdx.x; i <= C / a.group; i += NT) a.offsets[i] = (int)(i * rows);
}

// Any number of taps and channels: grid (rows, channels / 128), a thread per channel of a row.
template <typename T>
__global__ void __launch_bounds__(NT) conv_plain_kernel(ConvArgs a, int64_t rows) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t row = blockIdx.x, C = a.m.channels, ch = (int64_t)blockIdx.y * NT + threadIdx.x;
  if (a.offsets && a.group > 0 && row == 0 && blockIdx.y == 0)
    for (int64_t i = threadIdx.x; i <= C / a.group; i += NT) a.offsets[i] = (int)(i * rows);
  if (ch >= C) return;
  const int lane = row_lane(a.map, row), pos = row_pos(a.map, row), taps = a.m.taps, slots = taps - 1;
  if (pos < 0 || pos >= a.capacity) {
    if (ch == 0) atomicExch(a.status, KS_BAD_INDEX);
    return;
  }
  const int ahead = rows_ahead(a.map, row, lane, pos, slots);
  auto value = [&](int64_t r) {
    float v = a.m.in_bias ? a.m.in_bias[ch] : 0.f;
    for (int s = 0; s < a.nsplit; ++s) v += a.partial[s * a.split_stride + r * a.ld + ch];
    return v;
  };
  const float now = value(row);
  float y = a.m.bias ? a.m.bias[ch] : 0.f;
  for (int b = 0; b < taps; ++b) {
    float x = now;
    if (b > 0) x = b <= ahead ? value(row - b) : pos - b >= 0 ? a.state[((int64_t)lane * slots + (pos - b) % slots) * C + ch] : 0.f;
    y = fmaf(a.m.w[(taps - 1 - b) * C + ch], x, y);
  }
  if (!a.tails && slots > 0) a.state[((int64_t)lane * slots + pos % slots) * C + ch] = now;
  if (a.m.silu) y = silu_act(y);
  T* out = reinterpret_cast<T*>(a.out);
  if (a.group > 0) out[(ch / a.group * rows + row) * a.ldo + ch % a.group] = stf<T>(y);
  else out[row * a.ldo + ch] = stf<T>(y);
}

// The last inputs of every portion into the state.  grid (tails, channels / 128)
__global__ void __launch_bounds__(NT) conv_state_kernel(ConvArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int2 tail = a.tails[blockIdx.x];
  const int slots = a.m.taps - 1;
  if (tail.y >= slots) return;
  const int64_t C = a.m.channels, ch = (int64_t)blockIdx.y * NT + threadIdx.x;
  const int pos = row_pos(a.map, tail.x);
  if (ch >= C || pos < 0 || pos >= a.capacity) return;
  float v = a.m.in_bias ? a.m.in_bias[ch] : 0.f;
#pragma unroll 4
  for (int s = 0; s < a.nsplit; ++s) v += a.partial[s * a.split_stride + tail.x * a.ld + ch];
  a.state[((int64_t)row_lane(a.map, tail.x) * slots + pos % slots) * C + ch] = v;
}

}  // namespace

int conv_launch(Ctx* c, const ConvArgs& a, int64_t rows) {
  if (rows == 0) return REWB200_OK;
  const int64_t C = a.m.channels;
  const bool bf = a.dtype == REWB200_BF16;
  const bool vec = C % 4 == 0 && a.ld % 4 == 0 && a.ldo % 4 == 0 && a.group % 4 == 0 && a.split_stride % 4 == 0 &&
                   (reinterpret_cast<uintptr_t>(a.partial) & 15) == 0 && a.m.taps <= 8 && c->conv_impl != 1;
  if (vec) {
    const unsigned gy = (unsigned)((C + 4 * NT - 1) / (4 * NT));
    int tr = a.map.row_lane ? MAX_TR : 1;         // long walks, but eight CTAs for every SM
    while (tr > 1 && (rows + tr - 1) / tr * gy < 8 * c->sm_count) tr /= 2;
    const dim3 grid((unsigned)((rows + tr - 1) / tr), gy);
    auto go = [&](auto kernel) { return launch_k(kernel, grid, dim3(NT), 0, c->stream, c->use_pdl, a, rows, tr); };
    RB_CUDA(a.m.taps <= 4 ? (bf ? go(conv_kernel<bf16, 4>) : go(conv_kernel<float, 4>)) : (bf ? go(conv_kernel<bf16, 8>) : go(conv_kernel<float, 8>)));
  } else {
    const dim3 grid((unsigned)rows, (unsigned)((C + NT - 1) / NT));
    RB_CUDA(bf ? launch_k(conv_plain_kernel<bf16>, grid, dim3(NT), 0, c->stream, c->use_pdl, a, rows)
               : launch_k(conv_plain_kernel<float>, grid, dim3(NT), 0, c->stream, c->use_pdl, a, rows));
  }
  ++g_launch_total;
  if (!a.tails || a.n_tails == 0 || a.m.taps < 2) return REWB200_OK;
  RB_CUDA(launch_k(conv_state_kernel, dim3((unsigned)a.n_tails, (unsigned)((C + NT - 1) / NT)), dim3(NT), 0, c->stream, c->use_pdl, a));
  ++g_launch_total;
  return REWB200_OK;
}

}  // namespace rewb
