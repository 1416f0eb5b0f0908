// Kernels of gqa.cuh: the fused post-processing of the input projection, attention of decoded tokens and small portions
// on mma.sync, and plain kernels for f32 models and head sizes the tensor-core kernels do not take.  Norms, scores,
// biases, softmax and gates are f32 throughout.
#include <math.h>

#include <algorithm>

#include "gqa.cuh"
#include "ptx.cuh"

namespace rewb {

extern int64_t g_launch_total;

namespace {

constexpr int PAGE_TOKENS = 64;
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
__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }

__device__ __forceinline__ void add4(float4& v, float4 w) { v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w; }
__device__ __forceinline__ void fma4(float4& y, float4 w, float4 x) {
  y.x = fmaf(w.x, x.x, y.x);
  y.y = fmaf(w.y, x.y, y.y);
  y.z = fmaf(w.z, x.z, y.z);
  y.w = fmaf(w.w, x.w, y.w);
}
// Four neighbouring columns of a row that need not be aligned, summed over the slabs; columns past `n` read as zero.
__device__ __forceinline__ float4 slab4(const float* p, int nsplit, int64_t split_stride, int i, int n) {
  float e[4] = {0.f, 0.f, 0.f, 0.f};
  for (int u = 0; u < 4 && i + u < n; ++u)
    for (int s = 0; s < nsplit; ++s) e[u] += p[s * split_stride + i + u];
  return make_float4(e[0], e[1], e[2], e[3]);
}
__device__ __forceinline__ float4 slab4(const GqaPostArgs& a, const float* p, int i, int n) { return slab4(p, a.nsplit, a.split_stride, i, n); }
template <typename T>
__device__ __forceinline__ void put4(T* d, int i, int n, float4 v) {
  if (i >= n) return;
  if constexpr (sizeof(T) == 2) {
    if (i + 4 <= n && (reinterpret_cast<uintptr_t>(d + i) & 7) == 0) {
      *reinterpret_cast<uint2*>(d + i) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
      return;
    }
  }
  const float e[4] = {v.x, v.y, v.z, v.w};
  for (int u = 0; u < 4 && i + u < n; ++u) d[i + u] = stf<T>(e[u]);
}

// Rows of the same portion ahead of `row` in this step, at most taps - 1.
__device__ __forceinline__ int rows_ahead(const GqaPostArgs& a, int64_t row, int pos) {
  int n = 0;
  if (a.map.row_lane)
    while (n + 1 < a.m.taps && row - n - 1 >= 0 && a.map.row_lane[row - n - 1] == a.map.row_lane[row] && a.map.row_pos[row - n - 1] == pos - n - 1) ++n;
  return n;
}

constexpr int POST_ROWS = 8;       // rows a warp of gqa_post_kernel takes in large steps
constexpr int CONV_REG_TAPS = 4;   // convolutions up to this long run on registers

// One warp per head: query heads, key heads, value heads (none where the values are the keys: a key warp writes both), then
// one warp for all gates; RW rows each, requested together.  A lane holds four columns at a time, PC of them (dim and vdim up
// to 128 PC).  TIME: the head has a convolution, rotated features or values that are its keys (one row a warp; large steps:
// gqa_post_rows_kernel).
template <typename T, int PC, int RW, bool TIME>
__global__ void __launch_bounds__(256) gqa_post_kernel(GqaPostArgs a, int64_t rows) {
  static_assert(!TIME || RW == 1, "one row a warp");
  constexpr int HIST = TIME ? CONV_REG_TAPS - 1 : 0, BACK = TIME ? CONV_REG_TAPS : 1;
  constexpr unsigned ALL = 0xffffffffu;
  __shared__ __align__(16) float s_rot[TIME ? 8 : 1][TIME ? PC * 128 : 4];
  pdl_launch_dependents();
  const int64_t row0 = (int64_t)blockIdx.x * RW;
  const int nr = (int)min((int64_t)RW, rows - row0);
  const int unit = blockIdx.y * 8 + (threadIdx.x >> 5), ln = threadIdx.x & 31;
  const int H = a.m.heads, G = a.m.own_kv ? a.m.kv_heads : 0, K = a.m.dim, V = a.m.vdim, GV = TIME && a.m.v_from_k ? 0 : G;
  if (unit > H + G + GV || (unit == H + G + GV && !a.m.gate)) return;
  const bool is_q = unit < H, is_v = unit >= H + G;
  const int n = is_v ? V : K;
  const int64_t col = is_v ? (int64_t)(H + G) * K + (int64_t)(unit - H - G) * V : (int64_t)unit * K;
  const bool vec = col % 4 == 0 && n % 4 == 0 && a.ld % 4 == 0;
  // norm and convolution weights depend on no earlier kernel
  if (RW == 1 && a.m.q_norm) prefetch_floats(a.m.q_norm, K);
  if (RW == 1 && a.m.k_norm) prefetch_floats(a.m.k_norm, K);
  const int64_t C = TIME ? gqa_channels(a.m) : 0;
  const bool conv = TIME && a.m.taps > 0 && !is_v, conv_reg = conv && vec && a.m.taps <= CONV_REG_TAPS;
  const int half = TIME && !is_v ? a.m.rope_dims / 2 : 0;
  float4 cw[BACK][PC], past[BACK][PC];   // weights and values by tokens ago; past[0] is not used
  if constexpr (TIME) {
    if (conv_reg) {
#pragma unroll
      for (int b = 0; b < BACK; ++b)
#pragma unroll
        for (int c = 0; c < PC; ++c) {
          const int i = (c * 32 + ln) * 4;
          past[b][c] = make_float4(0.f, 0.f, 0.f, 0.f);
          cw[b][c] = b < a.m.taps && i < n ? *reinterpret_cast<const float4*>(a.m.conv + (a.m.taps - 1 - b) * C + col + i) : past[b][c];
        }
    }
  }
  if (!a.early) pdl_wait();
  // Lane l looks up row0 - HIST + l, in a captured decode step while the projection still runs.
  const int64_t my_row = row0 - HIST + ln;
  int my_lane = -1, my_pos = -1, my_page = 0;
  if (my_row >= 0 && my_row < row0 + nr && ln < RW + HIST) {
    my_lane = row_lane(a.map, my_row);
    my_pos = row_pos(a.map, my_row);
    const bool in = my_pos >= 0 && my_pos < a.capacity;
    my_page = a.block_table[(int64_t)my_lane * a.max_pages + (in ? my_pos / PAGE_TOKENS : 0)];
    if (!in && unit == 0 && ln >= HIST) atomicExch(a.status, KS_BAD_INDEX);
  }
  auto pos_of = [&](int r) { return __shfl_sync(ALL, my_pos, min(r, nr - 1) + HIST); };
  auto ok_at = [&](int pos) { return pos >= 0 && pos < a.capacity; };
  // which rows go on where the row ahead of them ended
  unsigned cont = 0;
  if constexpr (TIME) {
    const int pl = __shfl_up_sync(ALL, my_lane, 1), pp = __shfl_up_sync(ALL, my_pos, 1);
    cont = __ballot_sync(ALL, a.map.row_lane && ln > 0 && my_lane >= 0 && pl == my_lane && pp == my_pos - 1);
  }
  auto ahead_of = [&](int r) { return min(__clz(~(cont << (31 - HIST - r))), HIST); };   // rows of its portion ahead of row r in this step, at most HIST
  auto state_at = [&](int lane, int pos) -> float* { return a.state + ((int64_t)lane * (a.m.taps - 1) + pos % (a.m.taps - 1)) * C + col; };
  float4 t0 = make_float4(0.f, 0.f, 0.f, 0.f), t1 = t0;   // (cos, sin) of this lane's four features
  const bool rot_reg = PC == 1 && half > 0 && half % 4 == 0 && !a.m.pairs;
  auto rope_row = [&](int pos) { return a.m.rope + (int64_t)(ok_at(pos) ? pos : 0) * half; };
  auto rope_load = [&](int pos) {
    const int i = ln * 4;
    if (i >= 2 * half) return;
    const float2* cs = rope_row(pos) + (i < half ? i : i - half);
    t0 = *reinterpret_cast<const float4*>(cs);
    t1 = *reinterpret_cast<const float4*>(cs + 2);
  };
  if constexpr (TIME) {
    const int pos = pos_of(0);
    const int lane = __shfl_sync(ALL, my_lane, HIST);
    if (conv_reg && !a.map.row_lane)
#pragma unroll
      for (int b = 1; b < BACK; ++b)
#pragma unroll
        for (int c = 0; c < PC; ++c) {
          const int i = (c * 32 + ln) * 4;
          if (b < a.m.taps && pos - b >= 0 && i < n) past[b][c] = *reinterpret_cast<const float4*>(state_at(lane, pos - b) + i);
        }
    if (rot_reg) rope_load(pos);
  }
  if (a.early) pdl_wait();
  const float* p = a.partial + row0 * a.ld;
  if (unit == H + G + GV) {
    p += (int64_t)H * K + (int64_t)G * K + (int64_t)GV * V;
    for (int i = ln; i < nr * H; i += 32) {
      const int r = i / H, h = i % H;
      float z = 0.f;
      for (int s = 0; s < a.nsplit; ++s) z += p[s * a.split_stride + r * a.ld + h];
      a.gate[(row0 + r) * H + h] = sigmoid(z);
    }
    return;
  }
  float4 x[RW][PC];
  if (vec) {
#pragma unroll
    for (int r = 0; r < RW; ++r)
#pragma unroll
      for (int c = 0; c < PC; ++c) {
        const int i = (c * 32 + ln) * 4;
        x[r][c] = r < nr && i < n ? *reinterpret_cast<const float4*>(p + r * a.ld + col + i) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
    constexpr int SU = RW == 1 ? 8 / PC : 1;   // slabs requested together
    for (int s = 1; s < a.nsplit; s += SU) {
      float4 w[SU][RW][PC];
#pragma unroll
      for (int u = 0; u < SU; ++u)
#pragma unroll
        for (int r = 0; r < RW; ++r)
#pragma unroll
          for (int c = 0; c < PC; ++c) {
            const int i = (c * 32 + ln) * 4;
            w[u][r][c] = s + u < a.nsplit && r < nr && i < n ? *reinterpret_cast<const float4*>(p + (s + u) * a.split_stride + r * a.ld + col + i)
                                                             : make_float4(0.f, 0.f, 0.f, 0.f);
          }
#pragma unroll
      for (int u = 0; u < SU; ++u)
#pragma unroll
        for (int r = 0; r < RW; ++r)
#pragma unroll
          for (int c = 0; c < PC; ++c) add4(x[r][c], w[u][r][c]);
    }
  } else {
#pragma unroll
    for (int r = 0; r < RW; ++r)
#pragma unroll
      for (int c = 0; c < PC; ++c) x[r][c] = r < nr ? slab4(a, p + r * a.ld + col, (c * 32 + ln) * 4, n) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  if (a.m.in_bias) {
#pragma unroll
    for (int c = 0; c < PC; ++c) {
      const float4 b = slab4(a.m.in_bias + col, 1, 0, (c * 32 + ln) * 4, n);
#pragma unroll
      for (int r = 0; r < RW; ++r) add4(x[r][c], b);
    }
  }
  if constexpr (TIME) {
    if (conv_reg) {
      if (a.map.row_lane) {
        const int ahead = ahead_of(0);
#pragma unroll
        for (int b = 1; b < BACK; ++b)
#pragma unroll
          for (int c = 0; c < PC; ++c) {
            const int i = (c * 32 + ln) * 4;
            if (b > ahead || i >= n) continue;
            for (int s = 0; s < a.nsplit; ++s) add4(past[b][c], *reinterpret_cast<const float4*>(p + s * a.split_stride - b * a.ld + col + i));
          }
      }
      const int pos = pos_of(0), lane = __shfl_sync(ALL, my_lane, HIST);
      const int given = a.map.row_lane ? ahead_of(0) : HIST;   // values at hand; older ones are the state's
#pragma unroll
      for (int c = 0; c < PC; ++c) {
        const int i = (c * 32 + ln) * 4;
        const float4 u = x[0][c];
        float4 y = make_float4(cw[0][c].x * u.x, cw[0][c].y * u.y, cw[0][c].z * u.z, cw[0][c].w * u.w);
#pragma unroll
        for (int b = 1; b < BACK; ++b) {
          float4 h = past[b][c];
          if (b > given && b < a.m.taps && pos - b >= 0 && i < n) h = *reinterpret_cast<const float4*>(state_at(lane, pos - b) + i);
          fma4(y, cw[b][c], h);
        }
        x[0][c] = y;
        if (!a.tails && a.m.taps > 1 && i < n && ok_at(pos)) *reinterpret_cast<float4*>(state_at(lane, pos) + i) = u;
      }
    } else if (conv) {
      const int pos = pos_of(0), lane = __shfl_sync(ALL, my_lane, HIST), ahead = rows_ahead(a, row0, pos);
#pragma unroll
      for (int c = 0; c < PC; ++c) {
        const int i = (c * 32 + ln) * 4;
        const float4 u = x[0][c];
        float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int b = 0; b < a.m.taps; ++b) {
          const float4 w = slab4(a.m.conv + (a.m.taps - 1 - b) * C + col, 1, 0, i, n);
          if (b == 0) fma4(y, w, u);
          else if (b <= ahead) fma4(y, w, slab4(a, p - b * a.ld + col, i, n));
          else if (pos - b >= 0) fma4(y, w, slab4(state_at(lane, pos - b), 1, 0, i, n));
        }
        x[0][c] = y;
        if (!a.tails && a.m.taps > 1 && ok_at(pos)) put4<float>(state_at(lane, pos), i, n, u);
      }
    }
  }
  const float* w = is_v ? nullptr : is_q ? a.m.q_norm : a.m.k_norm;
  float4 g[PC];
#pragma unroll
  for (int c = 0; c < PC; ++c) {
    const int i = (c * 32 + ln) * 4;
    g[c] = make_float4(1.f, 1.f, 1.f, 1.f);
    if (w) g[c] = make_float4(i < n ? w[i] : 0.f, i + 1 < n ? w[i + 1] : 0.f, i + 2 < n ? w[i + 2] : 0.f, i + 3 < n ? w[i + 3] : 0.f);
  }
#pragma unroll
  for (int r = 0; r < RW; ++r) {
    if (r >= nr) break;
    const int pos = pos_of(r), page = __shfl_sync(ALL, my_page, r + HIST);
    float f = 1.f;
    if (w || (is_v && a.m.v_norm)) {
      float ss = 0.f;
#pragma unroll
      for (int c = 0; c < PC; ++c) ss += x[r][c].x * x[r][c].x + x[r][c].y * x[r][c].y + x[r][c].z * x[r][c].z + x[r][c].w * x[r][c].w;
      f = 1.0f / sqrtf(warp_sum(ss) / (float)n + a.eps);
    }
    if (is_q && a.m.temp_every > 0) f *= 1.0f + a.m.temp_coef * logf((float)((pos + 1) / a.m.temp_every + 1));
    T* dst;
    if (is_q) {
      dst = reinterpret_cast<T*>(a.q) + (row0 + r) * a.ldq + (int64_t)unit * K;
    } else {
      if (!ok_at(pos)) continue;
      const int64_t crow = ((int64_t)page * G + (is_v ? unit - H - G : unit - H)) * PAGE_TOKENS + pos % PAGE_TOKENS;
      dst = is_v ? reinterpret_cast<T*>(a.vc) + crow * a.ldv : reinterpret_cast<T*>(a.kc) + crow * a.ldk;
      if (TIME && !is_v && a.m.v_from_k)
#pragma unroll
        for (int c = 0; c < PC; ++c) put4<T>(reinterpret_cast<T*>(a.vc) + crow * a.ldv, (c * 32 + ln) * 4, n, x[r][c]);
    }
#pragma unroll
    for (int c = 0; c < PC; ++c) x[r][c] = make_float4(x[r][c].x * f * g[c].x, x[r][c].y * f * g[c].y, x[r][c].z * f * g[c].z, x[r][c].w * f * g[c].w);
    if constexpr (TIME) {
      if (rot_reg) {
        // the four features of a lane lie in one half; the other half is half / 4 lanes away
        const bool lo = ln * 4 < half;
        const int from = (lo ? ln + half / 4 : ln - half / 4) & 31;
        const float sg = lo ? -1.f : 1.f;
        const float4 e = x[r][0];
        const float4 o = make_float4(__shfl_sync(ALL, e.x, from), __shfl_sync(ALL, e.y, from), __shfl_sync(ALL, e.z, from), __shfl_sync(ALL, e.w, from));
        if (ln * 4 < 2 * half)
          x[r][0] = make_float4(e.x * t0.x + sg * (o.x * t0.y), e.y * t0.z + sg * (o.y * t0.w), e.z * t1.x + sg * (o.z * t1.y), e.w * t1.z + sg * (o.w * t1.w));
      } else if (half > 0 && a.m.pairs) {
        const float2* cs = rope_row(pos);
#pragma unroll
        for (int c = 0; c < PC; ++c) {
          const int i = (c * 32 + ln) * 2;     // this lane's first pair
          float4& e = x[r][c];
          if (i < half) {
            const float2 t = cs[i];
            e = make_float4(e.x * t.x - e.y * t.y, e.y * t.x + e.x * t.y, e.z, e.w);
          }
          if (i + 1 < half) {
            const float2 t = cs[i + 1];
            e = make_float4(e.x, e.y, e.z * t.x - e.w * t.y, e.w * t.x + e.z * t.y);
          }
        }
      } else if (half > 0) {
        float* s = s_rot[threadIdx.x >> 5];
        const float2* cs = rope_row(pos);
#pragma unroll
        for (int c = 0; c < PC; ++c) *reinterpret_cast<float4*>(s + (c * 32 + ln) * 4) = x[r][c];
        __syncwarp();
#pragma unroll
        for (int c = 0; c < PC; ++c) {
          float* e = reinterpret_cast<float*>(&x[r][c]);
#pragma unroll
          for (int u = 0; u < 4; ++u) {
            const int i = (c * 32 + ln) * 4 + u;
            if (i >= 2 * half) continue;
            const float2 t = cs[i < half ? i : i - half];
            e[u] = i < half ? e[u] * t.x - s[i + half] * t.y : e[u] * t.x + s[i - half] * t.y;
          }
        }
        __syncwarp();
      }
    }
#pragma unroll
    for (int c = 0; c < PC; ++c) put4<T>(dst, (c * 32 + ln) * 4, n, x[r][c]);
  }
}

// The same for large steps of heads with a convolution, rotation or values that are their keys, where `rows_post_ok`: a warp
// owns four columns a lane of one head and walks down tr rows with the last values in registers.
constexpr int MAX_TR = 32, ROWS_POST_MIN = 512;
template <typename T, bool NORM>     // NORM: RMS norms or a query temperature
__global__ void __launch_bounds__(256, 4) gqa_post_rows_kernel(GqaPostArgs a, int64_t rows, int tr) {
  constexpr unsigned ALL = 0xffffffffu;
  // per row: position (-1: outside the cache), row of its page's first head in the cache, rows of its portion ahead of it in
  // this step (up to three), lane
  __shared__ int4 info[MAX_TR];
  pdl_launch_dependents();
  const int64_t row0 = (int64_t)blockIdx.x * tr;
  const int nr = (int)min((int64_t)tr, rows - row0);
  const int unit = blockIdx.y * 8 + (threadIdx.x >> 5), ln = threadIdx.x & 31;
  const int H = a.m.heads, G = a.m.own_kv ? a.m.kv_heads : 0, K = a.m.dim, V = a.m.vdim, GV = a.m.v_from_k ? 0 : G;
  const bool is_q = unit < H, is_v = unit >= H + G, twice = !is_q && !is_v && a.m.v_from_k;   // twice: key and value
  const int n = is_v ? V : K, i = ln * 4, half = is_v ? 0 : a.m.rope_dims / 2;
  const bool on = i < n && unit < H + G + GV;
  const int64_t col = (is_v ? (int64_t)(H + G) * K + (int64_t)(unit - H - G) * V : (int64_t)unit * K) + i, C = gqa_channels(a.m);
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f), one = make_float4(1.f, 1.f, 1.f, 1.f);
  float4 cw[CONV_REG_TAPS];
#pragma unroll
  for (int b = 0; b < CONV_REG_TAPS; ++b) {
    cw[b] = b == 0 && (is_v || a.m.taps == 0) ? one : zero;
    if (on && !is_v && b < a.m.taps) cw[b] = *reinterpret_cast<const float4*>(a.m.conv + (a.m.taps - 1 - b) * C + col);
  }
  const float* w = is_v ? nullptr : is_q ? a.m.q_norm : a.m.k_norm;
  const bool normed = w || (is_v && a.m.v_norm);
  const float4 bias = a.m.in_bias && on ? make_float4(a.m.in_bias[col], a.m.in_bias[col + 1], a.m.in_bias[col + 2], a.m.in_bias[col + 3]) : zero;
  const float4 g = NORM && w && on ? make_float4(w[i], w[i + 1], w[i + 2], w[i + 3]) : one;
  pdl_wait();
  if ((int)threadIdx.x < nr) {
    const int64_t row = row0 + threadIdx.x;
    const int lane = row_lane(a.map, row), pos = row_pos(a.map, row);
    const bool in = pos >= 0 && pos < a.capacity;
    int ahead = 0;
    if (a.map.row_lane)
#pragma unroll
      for (int b = 1; b < CONV_REG_TAPS; ++b)
        if (row >= b && a.map.row_lane[row - b] == lane && a.map.row_pos[row - b] == pos - b) ahead = b;
    const int page = a.block_table[(int64_t)lane * a.max_pages + (in ? pos / PAGE_TOKENS : 0)];
    info[threadIdx.x] = make_int4(in ? pos : -1, page * G * PAGE_TOKENS + (in ? pos % PAGE_TOKENS : 0), ahead, lane);
    if (!in && blockIdx.y == 0) atomicExch(a.status, KS_BAD_INDEX);
  }
  __syncthreads();
  if (unit > H + G + GV || (unit == H + G + GV && !a.m.gate)) return;
  if (unit == H + G + GV) {
    const float* p = a.partial + row0 * a.ld + (int64_t)(H + G) * K + (int64_t)GV * V;
    for (int k = ln; k < nr * H; k += 32) {
      const int r = k / H, h = k % H;
      float z = 0.f;
      for (int s = 0; s < a.nsplit; ++s) z += p[s * a.split_stride + r * a.ld + h];
      a.gate[(row0 + r) * H + h] = sigmoid(z);
    }
    return;
  }
  auto value = [&](const float* p) {
    float4 v = on ? *reinterpret_cast<const float4*>(p) : zero;
    add4(v, bias);
    for (int s = 1; s < a.nsplit; ++s)
      if (on) add4(v, *reinterpret_cast<const float4*>(p + s * a.split_stride));
    return v;
  };
  auto state_at = [&](int lane, int pos) { return reinterpret_cast<float4*>(a.state + ((int64_t)lane * (a.m.taps - 1) + pos % (a.m.taps - 1)) * C + col); };
  const float* xp = a.partial + row0 * a.ld + col;
  float4 h1 = zero, h2 = zero, h3 = zero;   // projected values by tokens ago
  // those that no row at hand gives, from `first` tokens ago on
  auto from_state = [&](const int4& in, int first) {
    auto at = [&](int b) { return on && !is_v && b < a.m.taps && in.x - b >= 0 ? *state_at(in.w, in.x - b) : zero; };
    if (first <= 1) h1 = at(1);
    if (first <= 2) h2 = at(2);
    if (first <= 3) h3 = at(3);
  };
  from_state(info[0], info[0].z + 1);
  if (info[0].z >= 1) h1 = value(xp - a.ld);
  if (info[0].z >= 2) h2 = value(xp - 2 * a.ld);
  if (info[0].z >= 3) h3 = value(xp - 3 * a.ld);
  const bool lo = i < half, turned = i < 2 * half;
  const int from = (lo ? ln + half / 4 : ln - half / 4) & 31;
  const float sg = lo ? -1.f : 1.f;
  const float2* const rope = a.m.rope + (a.m.pairs ? i / 2 : lo ? i : i - half);
  const int hk = is_v ? unit - H - G : unit - H;
  T* const q = reinterpret_cast<T*>(a.q) + row0 * a.ldq + (int64_t)unit * K + i;
  T* const kc = reinterpret_cast<T*>(a.kc) + (int64_t)hk * PAGE_TOKENS * a.ldk + i;
  T* const vc = reinterpret_cast<T*>(a.vc) + (int64_t)hk * PAGE_TOKENS * a.ldv + i;
  const bool keep = !a.tails && a.m.taps > 1 && on && !is_v;
  auto put = [&](T* d, const float4& v) {
    if constexpr (sizeof(T) == 2) *reinterpret_cast<uint2*>(d) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
    else *reinterpret_cast<float4*>(d) = v;
  };
#pragma unroll 1
  for (int r = 0; r < nr; ++r) {
    const float4 x = value(xp);
    xp += a.ld;
    const int4 in = info[r];
    float4 t0, t1;
    if (turned) {
      const float2* cs = rope + (int64_t)max(in.x, 0) * half;
      t0 = *reinterpret_cast<const float4*>(cs);
      if (!a.m.pairs) t1 = *reinterpret_cast<const float4*>(cs + 2);
    }
    if (in.z == 0 && r > 0) from_state(in, 1);      // a portion starts here
    float4 y = make_float4(cw[0].x * x.x, cw[0].y * x.y, cw[0].z * x.z, cw[0].w * x.w);
    fma4(y, cw[1], h1);
    fma4(y, cw[2], h2);
    fma4(y, cw[3], h3);
    h3 = h2;
    h2 = h1;
    h1 = x;
    if (keep && in.x >= 0) *state_at(in.w, in.x) = x;
    if (twice && on && in.x >= 0) put(vc + (int64_t)in.y * a.ldv, y);
    if constexpr (NORM) {
      float f = 1.f;
      if (normed) f = 1.0f / sqrtf(warp_sum(y.x * y.x + y.y * y.y + y.z * y.z + y.w * y.w) / (float)n + a.eps);
      if (is_q && a.m.temp_every > 0) f *= 1.0f + a.m.temp_coef * logf((float)((in.x + 1) / a.m.temp_every + 1));
      y = make_float4(y.x * f * g.x, y.y * f * g.y, y.z * f * g.z, y.w * f * g.w);
    }
    if (half > 0 && a.m.pairs) {
      if (turned) y = make_float4(y.x * t0.x - y.y * t0.y, y.y * t0.x + y.x * t0.y, y.z * t0.z - y.w * t0.w, y.w * t0.z + y.z * t0.w);
    } else if (half > 0) {
      const float4 o = make_float4(__shfl_sync(ALL, y.x, from), __shfl_sync(ALL, y.y, from), __shfl_sync(ALL, y.z, from), __shfl_sync(ALL, y.w, from));
      if (turned) y = make_float4(y.x * t0.x + o.x * (sg * t0.y), y.y * t0.z + o.y * (sg * t0.w), y.z * t1.x + o.z * (sg * t1.y), y.w * t1.z + o.w * (sg * t1.w));
    }
    if (is_q) {
      if (on) put(q + r * a.ldq, y);
    } else if (on && in.x >= 0) {
      put(is_v ? vc + (int64_t)in.y * a.ldv : kc + (int64_t)in.y * a.ldk, y);
    }
  }
}
bool rows_post_ok(const GqaPostArgs& a) {
  const GqaDims& m = a.m;
  return m.dim <= 128 && m.vdim <= 128 && m.dim % 4 == 0 && m.vdim % 4 == 0 && a.ld % 4 == 0 && a.ldq % 4 == 0 && m.taps <= CONV_REG_TAPS && m.rope_dims % 8 == 0;
}

// The last values of every portion into the convolution state.  grid (tails, channels / 512)
__global__ void __launch_bounds__(128) gqa_conv_state_kernel(GqaPostArgs a) {
  pdl_launch_dependents();
  pdl_wait();
  const int2 tail = a.tails[blockIdx.x];
  const int slots = a.m.taps - 1;
  if (tail.y >= slots) return;
  const int64_t C = gqa_channels(a.m), i = ((int64_t)blockIdx.y * 128 + threadIdx.x) * 4;
  const int pos = row_pos(a.map, tail.x);
  if (i >= C || pos < 0 || pos >= a.capacity) return;
  const float* p = a.partial + tail.x * a.ld;
  float* s = a.state + ((int64_t)row_lane(a.map, tail.x) * slots + pos % slots) * C;
  if (C % 4 == 0 && a.ld % 4 == 0) {
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int k = 0; k < a.nsplit; ++k) {
      const float4 w = *reinterpret_cast<const float4*>(p + k * a.split_stride + i);
      v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w;
    }
    *reinterpret_cast<float4*>(s + i) = v;
  } else {
    put4<float>(s, (int)i, (int)C, slab4(a, p, (int)i, (int)C));
  }
}

// ------------------------------------------------------------------ plain attention: one CTA per (row of a tile, head),
// online softmax over 64-key pages
template <typename T>
__global__ void __launch_bounds__(128) gqa_plain_kernel(GqaAttnArgs a) {
  extern __shared__ float sm[];  // [dim] query, [vdim] accumulator, [64] scores
  pdl_launch_dependents();
  pdl_wait();
  const int2 tr = tile_rows(a.tiles, blockIdx.x / a.max_tile_rows);
  const int k_in = blockIdx.x % a.max_tile_rows;
  if (k_in >= tr.y) return;
  const int64_t row = tr.x + k_in;
  const int h = blockIdx.y, K = a.m.dim, V = a.m.vdim, G = a.m.kv_heads, hk = h / (a.m.heads / G);
  float *q = sm, *acc = sm + K, *sc = acc + V;
  const T* qp = reinterpret_cast<const T*>(a.q) + row * a.ldq + (int64_t)h * K;
  for (int i = threadIdx.x; i < K; i += 128) q[i] = ldf<T>(qp[i]);
  for (int i = threadIdx.x; i < V; i += 128) acc[i] = 0.f;
  const int lane = row_lane(a.map, row), pos = min(max(row_pos(a.map, row), 0), a.max_pages * PAGE_TOKENS - 1);
  const int w = threadIdx.x >> 5, ln = threadIdx.x & 31;
  const float* tab = a.m.bias ? a.m.bias + (int64_t)h * a.m.n_bias : nullptr;
  float mx = a.m.sink ? a.m.sink[h] : -INFINITY, l = a.m.sink ? 1.f : 0.f;
  __syncthreads();
  for (int t = 0; t <= pos / PAGE_TOKENS; ++t) {
    const int page = a.block_table[(int64_t)lane * a.max_pages + t];
    const T* kb = reinterpret_cast<const T*>(a.kc) + ((int64_t)page * G + hk) * PAGE_TOKENS * a.ldk;
    const T* vb = reinterpret_cast<const T*>(a.vc) + ((int64_t)page * G + hk) * PAGE_TOKENS * a.ldv;
    for (int j = w; j < PAGE_TOKENS; j += 4) {
      const int key = t * PAGE_TOKENS + j;
      float s = 0.f;
      if (key <= pos)
        for (int i = ln; i < K; i += 32) s = fmaf(q[i], ldf<T>(kb[(int64_t)j * a.ldk + i]), s);
      s = warp_sum(s);
      if (ln == 0) sc[j] = key <= pos ? s * a.m.scale + (tab ? tab[min(pos - key, a.m.n_bias - 1)] : 0.f) : -INFINITY;
    }
    __syncthreads();
    float tm = mx;
    for (int j = 0; j < PAGE_TOKENS; ++j) tm = fmaxf(tm, sc[j]);
    const float alpha = mx == -INFINITY ? 0.f : expf(mx - tm);
    __syncthreads();
    if (threadIdx.x < PAGE_TOKENS) sc[threadIdx.x] = sc[threadIdx.x] == -INFINITY ? 0.f : expf(sc[threadIdx.x] - tm);
    __syncthreads();
    float ps = 0.f;
    for (int j = 0; j < PAGE_TOKENS; ++j) ps += sc[j];
    l = l * alpha + ps;
    mx = tm;
    const int j1 = min(PAGE_TOKENS - 1, pos - t * PAGE_TOKENS);
    for (int i = threadIdx.x; i < V; i += 128) {
      float v = acc[i] * alpha;
      for (int j = 0; j <= j1; ++j) v = fmaf(sc[j], ldf<T>(vb[(int64_t)j * a.ldv + i]), v);
      acc[i] = v;
    }
    __syncthreads();
  }
  const float g = (a.m.gate ? a.gate[row * a.m.heads + h] : 1.0f) / l;
  T* op = reinterpret_cast<T*>(a.out) + row * a.ldo + (int64_t)h * V;
  for (int i = threadIdx.x; i < V; i += 128) op[i] = stf<T>(acc[i] * g);
}

// ------------------------------------------------------------------ bf16 on the tensor cores
// grid (kv splits, tiles * subtiles, kv heads * head groups), four consumer warps and a TMA warp.  A CTA's 16 rows are
// `heads_per` query heads of one kv head times `tokens_per` tokens; every K / V page is loaded once for all of them.
// Warp w owns keys 16 w .. 16 w + 15 of every page with a softmax state of its own in registers (no barrier between
// warps but the ring's); the warps meet after the last page.
struct GqaCfg {
  int nb_k, nb_v;     // 64-column boxes of a key / value row
  int stages;
  int heads_per, hgroups, tokens_per, subtiles;
};

// A head's sink in base 2, -inf without one.
__device__ __forceinline__ float sink_l2(const GqaDims& m, int h) { return m.sink ? m.sink[h] * LOG2E : -INFINITY; }

// KS: 16-feature steps of a key row, VG: 16-column groups of a value row.
template <int KS, int VG>
__global__ void __launch_bounds__(160, KS <= 8 ? 3 : 1) gqa_attn_kernel(const __grid_constant__ CUtensorMap tm_k, const __grid_constant__ CUtensorMap tm_v,
                                                       GqaAttnArgs a, GqaCfg cf) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int kb = cf.nb_k * 8192, stage_bytes = kb + cf.nb_v * 8192;
  uint8_t* sKV = smem;
  uint8_t* sQ = sKV + cf.stages * stage_bytes;                      // [box][16 rows][128 bytes]
  float* sM = reinterpret_cast<float*>(sQ + cf.nb_k * 2048);        // [4 warps][16] maxima, [4][16] sums
  uint64_t* full = reinterpret_cast<uint64_t*>(sM + 128);
  uint64_t* empty = full + 8;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l8 = lane & 7, lq = lane >> 3, g = lane >> 2, t = lane & 3;
  if (tid == 128) {
    for (int i = 0; i < cf.stages; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 4);
    }
    fence_barrier_init();
    tma_prefetch_desc(&tm_k);
    tma_prefetch_desc(&tm_v);
  }
  pdl_launch_dependents();
  {
    // bias tables and sinks depend on no earlier kernel
    const int group = a.m.heads / a.m.kv_heads, first = (int)blockIdx.z / cf.hgroups * group + ((int)blockIdx.z % cf.hgroups) * cf.heads_per;
    if (a.m.bias) prefetch_floats(a.m.bias + (int64_t)first * a.m.n_bias, min(cf.heads_per, a.m.heads - first) * a.m.n_bias);
    if (a.m.sink) prefetch_floats(a.m.sink + first, 1);
  }
  __syncthreads();
  if (!a.early_kv) pdl_wait();
  const int2 tr = tile_rows(a.tiles, (int)blockIdx.y / cf.subtiles);
  const int tok0 = ((int)blockIdx.y % cf.subtiles) * cf.tokens_per;
  const int ntok = min(cf.tokens_per, tr.y - tok0);
  if (ntok <= 0) return;
  const int64_t row0 = tr.x + tok0;
  const int hk = blockIdx.z / cf.hgroups, group = a.m.heads / a.m.kv_heads;
  const int hsub = ((int)blockIdx.z % cf.hgroups) * cf.heads_per, nh = min(cf.heads_per, group - hsub), head0 = hk * group + hsub;
  const int lane_id = row_lane(a.map, row0);
  const int cap = a.max_pages * PAGE_TOKENS;
  const int pos_first = min(max(row_pos(a.map, row0), 0), cap - 1), pos_last = min(pos_first + ntok - 1, cap - 1);
  const int nt_all = pos_last / PAGE_TOKENS + 1;
  const int per = (nt_all + (int)gridDim.x - 1) / (int)gridDim.x;
  const int t0 = (int)blockIdx.x * per, nt = max(0, min(per, nt_all - t0));
  if (warp == 4) {
    if (lane == 0) {
      auto load_page = [&](int i) {
        const int st = i % cf.stages;
        const int y = (a.block_table[(int64_t)lane_id * a.max_pages + t0 + i] * a.m.kv_heads + hk) * PAGE_TOKENS;
        mbar_expect_tx(&full[st], stage_bytes);
        for (int b = 0; b < cf.nb_k; ++b) tma_load_2d(sKV + st * stage_bytes + b * 8192, &tm_k, &full[st], b * 64, y);
        for (int b = 0; b < cf.nb_v; ++b) tma_load_2d(sKV + st * stage_bytes + kb + b * 8192, &tm_v, &full[st], b * 64, y);
      };
      int i = 0;
      if (a.early_kv) {
        const int newest = pos_last / PAGE_TOKENS - t0;   // the page the step's own row is written to
        for (; i < min(cf.stages, nt) && i < newest; ++i) load_page(i);
        pdl_wait();
      }
      for (; i < nt; ++i) {
        if (i >= cf.stages && !mbar_wait(&empty[i % cf.stages], ((i / cf.stages) - 1) & 1, a.status)) break;
        load_page(i);
      }
    }
    return;
  }
  if (a.early_kv) pdl_wait();
  auto consumers_sync = [] { asm volatile("bar.sync 1, 128;" ::: "memory"); };
  for (int i = tid; i < 16 * cf.nb_k * 8; i += 128) {
    const int m = i / (cf.nb_k * 8), c = i % (cf.nb_k * 8);
    const int tok = m / cf.heads_per, hh = m % cf.heads_per;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (tok < ntok && hh < nh && c * 8 < a.m.dim)   // dim is a multiple of 8
      v = *reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(a.q) + (row0 + tok) * a.ldq + (int64_t)(head0 + hh) * a.m.dim + c * 8);
    *reinterpret_cast<uint4*>(sQ + (c >> 3) * 2048 + swz128((uint32_t)m, (uint32_t)(c & 7))) = v;
  }
  consumers_sync();
  const int ks = (a.m.dim + 15) / 16, vg = (a.m.vdim + 15) / 16;
  uint32_t qf[KS][4];
  const uint32_t q_base = smem_u32(sQ);
#pragma unroll
  for (int k = 0; k < KS; ++k)
    if (k < ks)
      ldmatrix_x4(qf[k][0], qf[k][1], qf[k][2], qf[k][3], q_base + (k >> 2) * 2048 + swz128((lq & 1) * 8 + l8, (k & 3) * 2 + (lq >> 1)));
  const int rows_in = ntok * cf.heads_per;          // rows in use come first
  const int nr = rows_in > 8 ? 2 : 1;
  // this thread's rows: g and g + 8
  const float sl2 = a.m.scale * LOG2E;
  int spos[2];
  const float* tab[2];
  float far[2];
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    const int m = g + 8 * r, tok = m / cf.heads_per, hh = m % cf.heads_per;
    spos[r] = tok < ntok && hh < nh ? pos_first + tok : -1;   // -1: sees no key
    tab[r] = a.m.bias ? a.m.bias + (int64_t)(head0 + min(hh, nh - 1)) * a.m.n_bias : nullptr;
    far[r] = tab[r] ? tab[r][a.m.n_bias - 1] * LOG2E : 0.f;
  }
  float mrun[2] = {-INFINITY, -INFINITY}, lrun[2] = {0.f, 0.f};
  float acc[VG][2][4];
#pragma unroll
  for (int j = 0; j < VG; ++j)
#pragma unroll
    for (int e = 0; e < 8; ++e) acc[j][e >> 2][e & 3] = 0.f;
  uint32_t k_off[4], v_off[4];
#pragma unroll
  for (int u = 0; u < 4; ++u) {
    k_off[u] = swz128(warp * 16 + (lq >> 1) * 8 + l8, u * 2 + (lq & 1));
    v_off[u] = swz128(warp * 16 + (lq & 1) * 8 + l8, u * 2 + (lq >> 1));
  }
  const uint32_t kv_base = smem_u32(sKV);
  bool ok = true;
  for (int it = 0; it < nt; ++it) {
    const int st = it % cf.stages;
    if (ok) ok = mbar_wait(&full[st], (it / cf.stages) & 1, a.status);
    const uint32_t kp = kv_base + st * stage_bytes, vp = kp + kb;
    float sc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
#pragma unroll
    for (int k = 0; k < KS; ++k) {
      if (k >= ks) break;
      uint32_t b0, b1, b2, b3;
      ldmatrix_x4(b0, b1, b2, b3, kp + (k >> 2) * 8192 + k_off[k & 3]);
      mma_bf16_16816(sc[0], qf[k], b0, b1);
      mma_bf16_16816(sc[1], qf[k], b2, b3);
    }
    const int key0 = (t0 + it) * PAGE_TOKENS + warp * 16 + 2 * t;
    const bool inside = (t0 + it) * PAGE_TOKENS + PAGE_TOKENS - 1 <= pos_first - (a.m.bias ? a.m.n_bias - 1 : 0);   // every distance has the far bias
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        if ((e >> 1) >= nr) continue;
        const int r = e >> 1, dist = spos[r] - (key0 + n * 8 + (e & 1));
        float b = far[r];
        if (!inside && tab[r] && dist >= 0) b = __ldg(tab[r] + min(dist, a.m.n_bias - 1)) * LOG2E;
        sc[n][e] = dist >= 0 ? fmaf(sc[n][e], sl2, b) : -INFINITY;
        mx[r] = fmaxf(mx[r], sc[n][e]);
      }
    float alpha[2] = {1.f, 1.f}, muse[2] = {0.f, 0.f};
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      if (r >= nr) break;
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
      mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
      const float mn = fmaxf(mrun[r], mx[r]);
      muse[r] = mn == -INFINITY ? 0.f : mn;
      alpha[r] = ex2(mrun[r] - muse[r]);
      mrun[r] = mn;
    }
    uint32_t pf[4] = {0u, 0u, 0u, 0u};
    float ps[2] = {0.f, 0.f};
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        if (r >= nr) break;
        const float p0 = ex2(sc[n][2 * r] - muse[r]), p1 = ex2(sc[n][2 * r + 1] - muse[r]);
        ps[r] += p0 + p1;
        pf[n * 2 + r] = pack_bf16(p0, p1);
      }
    lrun[0] = lrun[0] * alpha[0] + ps[0];
    lrun[1] = lrun[1] * alpha[1] + ps[1];
    if (__any_sync(0xffffffffu, alpha[0] != 1.f || alpha[1] != 1.f)) {
#pragma unroll
      for (int j = 0; j < VG; ++j)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          acc[j][n][0] *= alpha[0];
          acc[j][n][1] *= alpha[0];
          if (nr > 1) {
            acc[j][n][2] *= alpha[1];
            acc[j][n][3] *= alpha[1];
          }
        }
    }
#pragma unroll
    for (int j = 0; j < VG; ++j) {
      if (j >= vg) break;
      uint32_t v0, v1, v2, v3;
      ldmatrix_x4_trans(v0, v1, v2, v3, vp + (j >> 2) * 8192 + v_off[j & 3]);
      mma_bf16_16816(acc[j][0], pf, v0, v1);
      mma_bf16_16816(acc[j][1], pf, v2, v3);
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[st]);
  }
#pragma unroll
  for (int r = 0; r < 2; ++r) {
    lrun[r] += __shfl_xor_sync(0xffffffffu, lrun[r], 1);
    lrun[r] += __shfl_xor_sync(0xffffffffu, lrun[r], 2);
    if (t == 0) {
      sM[warp * 16 + g + 8 * r] = mrun[r];
      sM[64 + warp * 16 + g + 8 * r] = lrun[r];
    }
  }
  // the stages are read out: they hold the warps' accumulators now, [4][16][vg * 16 + 4]
  consumers_sync();
  float* sO = reinterpret_cast<float*>(sKV);
  const int ldO = vg * 16 + 4;
#pragma unroll
  for (int j = 0; j < VG; ++j) {
    if (j >= vg) break;
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int r = 0; r < 2; ++r)
        if (g + 8 * r < rows_in) *reinterpret_cast<float2*>(sO + (warp * 16 + g + 8 * r) * ldO + j * 16 + n * 8 + 2 * t) = make_float2(acc[j][n][2 * r], acc[j][n][2 * r + 1]);
  }
  consumers_sync();
  const int V = a.m.vdim;   // a multiple of 8
  const bool last = gridDim.x == 1;
  for (int mrow = warp; mrow < rows_in; mrow += 4) {
    const int tok = mrow / cf.heads_per, hh = mrow - tok * cf.heads_per;
    if (hh >= nh) continue;
    const int h = head0 + hh;
    const int64_t row = row0 + tok;
    float mw[4], M = last ? sink_l2(a.m, h) : -INFINITY;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      mw[w] = sM[w * 16 + mrow];
      M = fmaxf(M, mw[w]);
    }
    const float mu = M == -INFINITY ? 0.f : M;
    float l = 0.f;
#pragma unroll
    for (int w = 0; w < 4; ++w) {
      mw[w] = ex2(mw[w] - mu);
      l += mw[w] * sM[64 + w * 16 + mrow];
    }
    float inv = 1.f;
    const int64_t u = (row * a.m.heads + h) * a.kv_splits + blockIdx.x;
    if (last) {
      if (a.m.sink) l += ex2(sink_l2(a.m, h) - mu);
      inv = (a.m.gate ? a.gate[row * a.m.heads + h] : 1.0f) / l;
    } else if (lane == 0) {
      a.ml[u] = make_float2(M, l);
    }
    for (int c = lane * 4; c < V; c += 128) {
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
      for (int w = 0; w < 4; ++w) {
        const float4 x = *reinterpret_cast<const float4*>(sO + (w * 16 + mrow) * ldO + c);
        o.x += mw[w] * x.x; o.y += mw[w] * x.y; o.z += mw[w] * x.z; o.w += mw[w] * x.w;
      }
      if (last)
        *reinterpret_cast<uint2*>(reinterpret_cast<bf16*>(a.out) + row * a.ldo + (int64_t)h * V + c) =
            make_uint2(pack_bf16(o.x * inv, o.y * inv), pack_bf16(o.z * inv, o.w * inv));
      else
        *reinterpret_cast<float4*>(a.o_part + u * V + c) = o;
    }
  }
}

// One warp per (row of a tile, head): the kv splits, the sink and the gate.
__global__ void __launch_bounds__(256) gqa_merge_kernel(GqaAttnArgs a) {
  pdl_launch_dependents();
  const int64_t u = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int ln = threadIdx.x & 31, H = a.m.heads, V = a.m.vdim, ns = a.kv_splits;
  const int64_t slot = u / H;
  const int h = (int)(u % H);
  if (slot >= (int64_t)a.tiles.count * a.max_tile_rows) return;
  pdl_wait();
  const int2 tr = tile_rows(a.tiles, (int)(slot / a.max_tile_rows));
  const int k = (int)(slot % a.max_tile_rows);
  if (k >= tr.y) return;
  const int64_t row = tr.x + k, at = (row * H + h) * ns;
  const float2 e = ln < ns ? a.ml[at + ln] : make_float2(-INFINITY, 0.f);   // at most 32 splits
  float M = e.x;
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
  const float sk = sink_l2(a.m, h);
  M = fmaxf(M, sk);
  const float mu = M == -INFINITY ? 0.f : M;
  const float f = ex2(e.x - mu);
  float l = warp_sum(f * e.y);
  if (a.m.sink) l += ex2(sk - mu);
  const float inv = (a.m.gate ? a.gate[row * H + h] : 1.0f) / l;
  for (int c0 = 0; c0 < V; c0 += 128) {
    const int c = c0 + ln * 4;
    float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int s = 0; s < ns; ++s) {
      const float w = __shfl_sync(0xffffffffu, f, s);
      if (c < V) {
        const float4 x = *reinterpret_cast<const float4*>(a.o_part + (at + s) * V + c);
        o.x += w * x.x; o.y += w * x.y; o.z += w * x.z; o.w += w * x.w;
      }
    }
    if (c < V)
      *reinterpret_cast<uint2*>(reinterpret_cast<bf16*>(a.out) + row * a.ldo + (int64_t)h * V + c) =
          make_uint2(pack_bf16(o.x * inv, o.y * inv), pack_bf16(o.z * inv, o.w * inv));
  }
}

bool mma_ok(const GqaDims& m) { return m.dim % 8 == 0 && m.vdim % 8 == 0 && m.dim <= 256 && m.vdim <= 256; }

GqaCfg config(const GqaDims& m, int max_tile_rows) {
  GqaCfg cf;
  const int group = m.heads / m.kv_heads;
  cf.nb_k = (m.dim + 63) / 64;
  cf.nb_v = (m.vdim + 63) / 64;
  cf.heads_per = std::min(group, 16);
  cf.hgroups = (group + cf.heads_per - 1) / cf.heads_per;
  cf.tokens_per = std::min(max_tile_rows, std::max(1, 16 / cf.heads_per));
  cf.subtiles = (max_tile_rows + cf.tokens_per - 1) / cf.tokens_per;
  cf.stages = std::min(4, std::max(2, (int)(64 * 1024 / ((cf.nb_k + cf.nb_v) * 8192))));
  return cf;
}

}  // namespace

int gqa_post_launch(Ctx* c, const GqaPostArgs& a, int64_t rows) {
  if (rows == 0) return REWB200_OK;
  const int units = a.m.heads + (a.m.own_kv ? (a.m.v_from_k ? 1 : 2) * a.m.kv_heads : 0) + (a.m.gate ? 1 : 0);
  const bool time = a.m.taps > 0 || a.m.rope_dims > 0 || a.m.v_from_k;
  RB_REQUIRE(a.m.dim <= 512 && a.m.vdim <= 512, "grouped-query attention: head sizes above 512");
  const bool small = a.m.dim <= 128 && a.m.vdim <= 128, bf = a.dtype == REWB200_BF16, many = small && bf && rows >= 512 && !time;
  const dim3 grid((unsigned)(many ? (rows + POST_ROWS - 1) / POST_ROWS : rows), (unsigned)((units + 7) / 8));
  auto go = [&](auto kernel) { return launch_k(kernel, grid, dim3(256), 0, c->stream, c->use_pdl, a, rows); };
  if (time && rows >= ROWS_POST_MIN && rows_post_ok(a)) {
    int tr = MAX_TR;         // long walks, but four CTAs for every SM
    while (tr > 4 && (rows + tr - 1) / tr * grid.y < 4 * c->sm_count) tr /= 2;
    const dim3 g((unsigned)((rows + tr - 1) / tr), grid.y);
    const bool norm = a.m.q_norm || a.m.k_norm || a.m.temp_every > 0 || a.m.v_norm;
    auto go_rows = [&](auto kernel) { return launch_k(kernel, g, dim3(256), 0, c->stream, c->use_pdl, a, rows, tr); };
    RB_CUDA(bf ? (norm ? go_rows(gqa_post_rows_kernel<bf16, true>) : go_rows(gqa_post_rows_kernel<bf16, false>))
               : (norm ? go_rows(gqa_post_rows_kernel<float, true>) : go_rows(gqa_post_rows_kernel<float, false>)));
    ++g_launch_total;
    return REWB200_OK;
  }
#define RB_POST(TIME)                                                                                      \
  (bf ? (small ? go(gqa_post_kernel<bf16, 1, 1, TIME>) : go(gqa_post_kernel<bf16, 4, 1, TIME>))            \
   : small ? go(gqa_post_kernel<float, 1, 1, TIME>) : go(gqa_post_kernel<float, 4, 1, TIME>))
  RB_CUDA(many ? go(gqa_post_kernel<bf16, 1, POST_ROWS, false>) : time ? RB_POST(true) : RB_POST(false));
#undef RB_POST
  ++g_launch_total;
  return REWB200_OK;
}

int gqa_conv_state_launch(Ctx* c, const GqaPostArgs& a) {
  if (a.n_tails == 0 || a.m.taps < 2) return REWB200_OK;
  const dim3 grid((unsigned)a.n_tails, (unsigned)((gqa_channels(a.m) + 511) / 512));
  RB_CUDA(launch_k(gqa_conv_state_kernel, grid, dim3(128), 0, c->stream, c->use_pdl, a));
  ++g_launch_total;
  return REWB200_OK;
}

// KV splits of a launch over `tiles` row tiles: enough CTAs for two per SM, no more than a split per page.
int gqa_kv_splits(Ctx* c, const GqaDims& m, int64_t tiles, int64_t max_ctx) {
  const int group = m.heads / m.kv_heads;
  const int64_t ctas = std::max<int64_t>(1, tiles * m.kv_heads * ((group + 15) / 16)), pages = (max_ctx + PAGE_TOKENS - 1) / PAGE_TOKENS;
  return (int)std::max<int64_t>(1, std::min<int64_t>({(2 * c->sm_count + ctas - 1) / ctas, pages, 16}));
}

int gqa_attn_launch(Ctx* c, const GqaAttnArgs& a) {
  if (a.tiles.count == 0) return REWB200_OK;
  if (a.dtype != REWB200_BF16 || c->gqa_impl == 1 || !mma_ok(a.m)) {
    const dim3 grid((unsigned)a.tiles.count * a.max_tile_rows, (unsigned)a.m.heads);
    const size_t smem = (a.m.dim + a.m.vdim + PAGE_TOKENS) * sizeof(float);
    RB_CUDA(a.dtype == REWB200_BF16 ? launch_k(gqa_plain_kernel<bf16>, grid, dim3(128), smem, c->stream, c->use_pdl, a)
                                    : launch_k(gqa_plain_kernel<float>, grid, dim3(128), smem, c->stream, c->use_pdl, a));
    ++g_launch_total;
    return REWB200_OK;
  }
  const GqaCfg cf = config(a.m, a.max_tile_rows);
  const size_t kv = (size_t)cf.stages * (cf.nb_k + cf.nb_v) * 8192, merge = (size_t)64 * ((a.m.vdim + 15) / 16 * 16 + 4) * 4;
  const size_t smem = std::max(kv, (merge + 1023) / 1024 * 1024) + cf.nb_k * 2048 + 512 + 256 + 1024;
  RB_REQUIRE(kv >= merge, "grouped-query attention: value heads too large for the merge buffer");
  const dim3 grid((unsigned)a.kv_splits, (unsigned)(a.tiles.count * cf.subtiles), (unsigned)(a.m.kv_heads * cf.hgroups));
  const int ks = (a.m.dim + 15) / 16, vg = (a.m.vdim + 15) / 16;
  auto go = [&](auto kernel) -> int {
    RB_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    RB_CUDA(launch_k(kernel, grid, dim3(160), smem, c->stream, c->use_pdl, *a.tm_k, *a.tm_v, a, cf));
    ++g_launch_total;
    return REWB200_OK;
  };
  if (ks <= 4 && vg <= 4) RB_TRY(go(gqa_attn_kernel<4, 4>));
  else if (ks <= 8 && vg <= 8) RB_TRY(go(gqa_attn_kernel<8, 8>));
  else RB_TRY(go(gqa_attn_kernel<16, 16>));
  if (a.kv_splits == 1) return REWB200_OK;
  const int64_t units = (int64_t)a.tiles.count * a.max_tile_rows * a.m.heads;
  RB_CUDA(launch_k(gqa_merge_kernel, dim3((unsigned)((units + 7) / 8)), dim3(256), 0, c->stream, c->use_pdl, a));
  ++g_launch_total;
  return REWB200_OK;
}

}  // namespace rewb
