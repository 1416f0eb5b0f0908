// Latent attention kernels (see latent.cuh): the fused post-processing of the input projection, and attention on the
// cached latents.  Scores, softmax, norms, rotations and gates are f32 throughout.
#include <math.h>

#include <algorithm>

#include "latent.cuh"
#include "ptx.cuh"

namespace rewb {

extern int64_t g_launch_total;

namespace {

constexpr int PAGE_TOKENS = 64;

__device__ __forceinline__ float2 rotate(float2 v, float2 cs) {
  return make_float2(v.x * cs.x - v.y * cs.y, v.y * cs.x + v.x * cs.y);
}

__device__ __forceinline__ void add4(float4& v, const float4 w) { v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w; }

// Sums of two values over the block; every thread gets both.
__device__ __forceinline__ float2 block_sum2(float2 v, float2* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    v.x += __shfl_xor_sync(0xffffffffu, v.x, o);
    v.y += __shfl_xor_sync(0xffffffffu, v.y, o);
  }
  if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
  __syncthreads();
  float2 t = make_float2(0.f, 0.f);
  for (int i = 0; i < (int)(blockDim.x >> 5); ++i) {
    t.x += red[i].x;
    t.y += red[i].y;
  }
  return t;
}

// One CTA per row; small steps (SMALL) have a thread per four columns, up to 768, and many slabs.
template <typename T, bool SMALL>
__global__ void __launch_bounds__(SMALL ? 768 : 128, SMALL ? 1 : 10) latent_post_kernel(LatentPostArgs a) {
  extern __shared__ __align__(16) float sx[];
  __shared__ float2 red[32];
  pdl_launch_dependents();
  const int64_t row = blockIdx.x;
  const int nt = blockDim.x;
  const int nq = a.m.q_rank, nc = a.m.own_kv ? a.m.kv_rank : 0, nr = a.m.own_kv ? a.m.rot_dim : 0, n = nq + nc + nr + (a.m.gate ? a.m.heads : 0);
  // the norm weights depend on no earlier kernel; in a captured decode step neither do the position and its table row
  if ((int)threadIdx.x * 32 < nq) prefetch_l2(a.q_norm + threadIdx.x * 32);
  if ((int)threadIdx.x * 32 < nc) prefetch_l2(a.kv_norm + threadIdx.x * 32);
  if (!a.early) pdl_wait();
  const int lane = row_lane(a.map, row), pos = row_pos(a.map, row);
  const bool ok = pos >= 0 && pos < a.capacity && pos < a.m.max_pos;
  if (a.early) {
    if (ok && a.m.rope_dims > 0 && (int)threadIdx.x * 32 < a.m.rope_dims) prefetch_l2(a.m.rope + (int64_t)pos * (a.m.rope_dims / 2) + threadIdx.x * 16);
    pdl_wait();
  }
  const float* p = a.partial + row * a.ld;
  float2 sq = make_float2(0.f, 0.f);
  for (int i = threadIdx.x * 4; i < n; i += nt * 4) {   // rows are padded to a multiple of 8 columns
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    if constexpr (SMALL) {
      for (int k = 0; k < a.nsplit; k += 8) {
        float4 w[8];
#pragma unroll
        for (int u = 0; u < 8; ++u)
          w[u] = k + u < a.nsplit ? *reinterpret_cast<const float4*>(p + (k + u) * a.split_stride + i) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int u = 0; u < 8; ++u) add4(v, w[u]);
      }
    } else {
      for (int k = 0; k < a.nsplit; ++k) add4(v, *reinterpret_cast<const float4*>(p + k * a.split_stride + i));
    }
    *reinterpret_cast<float4*>(sx + i) = v;
    const float e[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      if (i + u < nq) sq.x += e[u] * e[u];
      else if (i + u < nq + nc) sq.y += e[u] * e[u];
    }
  }
  const int page = a.block_table[(int64_t)lane * a.max_pages + (ok ? pos / PAGE_TOKENS : 0)];
  sq = block_sum2(sq, red);
  const float rq = 1.0f / sqrtf(sq.x / (float)nq + a.eps), rc = 1.0f / sqrtf(sq.y / (float)max(nc, 1) + a.eps);
  if (!ok && threadIdx.x == 0) atomicExch(a.status, KS_BAD_INDEX);
  T* cq = reinterpret_cast<T*>(a.cq) + row * a.ldcq;
  T* cr = reinterpret_cast<T*>(a.cache) + ((int64_t)page * PAGE_TOKENS + (ok ? pos % PAGE_TOKENS : 0)) * a.ldc;
  // two columns a thread: the pairs of the query latent, of the key/value latent and of the rotated part
  auto put = [](T* d, float x, float y) {
    if constexpr (sizeof(T) == 2) {
      if ((reinterpret_cast<uintptr_t>(d) & 3) == 0) {
        *reinterpret_cast<uint32_t*>(d) = pack_bf16(x, y);
        return;
      }
    }
    d[0] = stf<T>(x);
    d[1] = stf<T>(y);
  };
  for (int i = threadIdx.x * 2; i < nq; i += nt * 2) {
    if (i + 1 < nq) put(cq + i, a.q_norm[i] * (sx[i] * rq), a.q_norm[i + 1] * (sx[i + 1] * rq));
    else cq[i] = stf<T>(a.q_norm[i] * (sx[i] * rq));
  }
  if (a.m.gate)
    for (int i = threadIdx.x; i < a.m.heads; i += nt) a.gate[row * a.m.heads + i] = 1.0f / (1.0f + expf(-sx[nq + nc + nr + i]));
  if (!ok || !a.m.own_kv) return;
  for (int i = threadIdx.x * 2; i < nc; i += nt * 2) {
    if (i + 1 < nc) put(cr + i, a.kv_norm[i] * (sx[nq + i] * rc), a.kv_norm[i + 1] * (sx[nq + i + 1] * rc));
    else cr[i] = stf<T>(a.kv_norm[i] * (sx[nq + i] * rc));
  }
  const int half = a.m.rope_dims / 2;
  for (int i = threadIdx.x; i < half; i += nt) {
    const float2 v = rotate(make_float2(sx[nq + nc + 2 * i], sx[nq + nc + 2 * i + 1]), a.m.rope[(int64_t)pos * half + i]);
    put(cr + nc + 2 * i, v.x, v.y);
  }
  for (int i = 2 * half + threadIdx.x; i < nr; i += nt) cr[nc + i] = stf<T>(sx[nq + nc + i]);
}

// Large steps: a warp per row, which it holds in registers, four columns at a time (up to 128 NV; the parts of a row are
// multiples of four columns wide).
template <typename T, int NV>
__global__ void __launch_bounds__(256, NV <= 10 ? 3 : 2) latent_post_rows_kernel(LatentPostArgs a, int64_t rows) {
  pdl_launch_dependents();
  const int64_t row = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  const int ln = threadIdx.x & 31;
  if (row >= rows) return;
  const int nq = a.m.q_rank, nc = a.m.own_kv ? a.m.kv_rank : 0, nr = a.m.own_kv ? a.m.rot_dim : 0, n = nq + nc + nr + (a.m.gate ? a.m.heads : 0);
  pdl_wait();
  const float* p = a.partial + row * a.ld;
  float4 v[NV];
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = (k * 32 + ln) * 4;
    v[k] = i < n ? *reinterpret_cast<const float4*>(p + i) : make_float4(0.f, 0.f, 0.f, 0.f);   // rows are padded to a multiple of 8 columns
  }
  const int lane = row_lane(a.map, row), pos = row_pos(a.map, row);
  const bool ok = pos >= 0 && pos < a.capacity && pos < a.m.max_pos;
  const int page = a.block_table[(int64_t)lane * a.max_pages + (ok ? pos / PAGE_TOKENS : 0)];
  if (!ok && ln == 0) atomicExch(a.status, KS_BAD_INDEX);
  for (int s = 1; s < a.nsplit; ++s)
#pragma unroll
    for (int k = 0; k < NV; ++k) {
      const int i = (k * 32 + ln) * 4;
      if (i < n) add4(v[k], *reinterpret_cast<const float4*>(p + s * a.split_stride + i));
    }
  float sq = 0.f, sc = 0.f;
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = (k * 32 + ln) * 4;
    const float t = v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
    if (i < nq) sq += t;
    else if (i < nq + nc) sc += t;
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    sq += __shfl_xor_sync(0xffffffffu, sq, o);
    sc += __shfl_xor_sync(0xffffffffu, sc, o);
  }
  const float rq = 1.0f / sqrtf(sq / (float)nq + a.eps), rc = 1.0f / sqrtf(sc / (float)max(nc, 1) + a.eps);
  auto put = [](T* d, float4 y) {
    if constexpr (sizeof(T) == 2) *reinterpret_cast<uint2*>(d) = make_uint2(pack_bf16(y.x, y.y), pack_bf16(y.z, y.w));
    else *reinterpret_cast<float4*>(d) = y;
  };
  auto normed = [](const float* w, float4 x, float r) {
    const float4 g = *reinterpret_cast<const float4*>(w);
    return make_float4(g.x * (x.x * r), g.y * (x.y * r), g.z * (x.z * r), g.w * (x.w * r));
  };
  T* cq = reinterpret_cast<T*>(a.cq) + row * a.ldcq;
  T* cr = reinterpret_cast<T*>(a.cache) + ((int64_t)page * PAGE_TOKENS + (ok ? pos % PAGE_TOKENS : 0)) * a.ldc;
  const int half = a.m.rope_dims / 2;
#pragma unroll
  for (int k = 0; k < NV; ++k) {
    const int i = (k * 32 + ln) * 4;
    if (i >= n) break;
    if (i < nq) {
      put(cq + i, normed(a.q_norm + i, v[k], rq));
    } else if (i < nq + nc) {
      if (ok) put(cr + i - nq, normed(a.kv_norm + i - nq, v[k], rc));
    } else if (i < nq + nc + nr) {
      const int f = i - nq - nc;
      float4 y = v[k];
      const float2* cs = a.m.rope + (int64_t)(ok ? pos : 0) * half + f / 2;
      if (f < 2 * half) {
        const float2 t = rotate(make_float2(y.x, y.y), cs[0]);
        y.x = t.x;
        y.y = t.y;
      }
      if (f + 2 < 2 * half) {
        const float2 t = rotate(make_float2(y.z, y.w), cs[1]);
        y.z = t.x;
        y.w = t.y;
      }
      if (ok) put(cr + nc + f, y);
    } else {
      const float e[4] = {v[k].x, v[k].y, v[k].z, v[k].w};
      for (int u = 0; u < 4 && i + u < n; ++u) a.gate[row * a.m.heads + i + u - nq - nc - nr] = 1.0f / (1.0f + expf(-e[u]));
    }
  }
}

// ------------------------------------------------------------------ plain kernels (f32 models, and shapes the
// tensor-core kernels do not take): one CTA per (row of a tile, head)

__device__ __forceinline__ bool tile_row(const RowTiles& t, int per_tile, int64_t& row) {
  const int2 tr = tile_rows(t, blockIdx.x / per_tile);
  const int k = blockIdx.x % per_tile;
  row = tr.x + k;
  return k < tr.y;
}

template <typename T>
__device__ __forceinline__ float q_at(const LatentAttnArgs& a, int64_t row, int64_t col) {
  if (a.nsplit == 0) return ldf<T>(reinterpret_cast<const T*>(a.q)[row * a.ldq + col]);
  float v = 0.f;
  for (int s = 0; s < a.nsplit; ++s) v += reinterpret_cast<const float*>(a.q)[s * a.split_stride + row * a.ldq + col];
  return v;
}

// qeff[row][head] = [W_uk^T q_nope | rotated q_rot]
template <typename T>
__global__ void __launch_bounds__(128) latent_q_plain_kernel(LatentAttnArgs a) {
  extern __shared__ float sq[];
  pdl_launch_dependents();
  pdl_wait();
  int64_t row;
  if (!tile_row(a.tiles, a.max_tile_rows, row)) return;
  const int h = blockIdx.y, dn = a.m.dim, dr = a.m.rot_dim, r = a.m.kv_rank;
  for (int i = threadIdx.x; i < dn + dr; i += 128) sq[i] = ldf<T>(stf<T>(q_at<T>(a, row, (int64_t)h * (dn + dr) + i)));
  __syncthreads();
  T* qe = reinterpret_cast<T*>(a.qeff) + (row * a.m.heads + h) * a.ldc;
  const T* w = reinterpret_cast<const T*>(a.ukv) + (int64_t)h * dn;
  for (int k = threadIdx.x; k < r; k += 128) {
    float acc = 0.f;
    for (int i = 0; i < dn; ++i) acc = fmaf(sq[i], ldf<T>(w[(int64_t)k * a.ld_ukv + i]), acc);
    qe[k] = stf<T>(acc);
  }
  const int half = a.m.rope_dims / 2, pos = min(max(row_pos(a.map, row), 0), a.m.max_pos - 1);
  for (int i = threadIdx.x; i < half; i += 128) {
    const float2 v = rotate(make_float2(sq[dn + 2 * i], sq[dn + 2 * i + 1]), a.m.rope[(int64_t)pos * half + i]);
    qe[r + 2 * i] = stf<T>(v.x);
    qe[r + 2 * i + 1] = stf<T>(v.y);
  }
  for (int i = 2 * half + threadIdx.x; i < dr; i += 128) qe[r + i] = stf<T>(sq[dn + i]);
}

// Attention over the cache rows, online softmax over 64-key tiles.
template <typename T>
__global__ void __launch_bounds__(128) latent_attn_plain_kernel(LatentAttnArgs a) {
  extern __shared__ float sm[];  // [r + dr] query, [r] accumulator, [64] scores
  pdl_launch_dependents();
  pdl_wait();
  int64_t row;
  if (!tile_row(a.tiles, a.max_tile_rows, row)) return;
  const int h = blockIdx.y, r = a.m.kv_rank, dt = r + a.m.rot_dim;
  float* q = sm;
  float* acc = sm + dt;
  float* sc = acc + r;
  const T* qe = reinterpret_cast<const T*>(a.qeff) + (row * a.m.heads + h) * a.ldc;
  for (int i = threadIdx.x; i < dt; i += 128) q[i] = ldf<T>(qe[i]);
  for (int i = threadIdx.x; i < r; i += 128) acc[i] = 0.f;
  const int lane = row_lane(a.map, row), pos = min(max(row_pos(a.map, row), 0), a.max_pages * PAGE_TOKENS - 1);
  const int k0 = a.m.window > 0 ? max(0, pos - a.m.window + 1) : 0;
  const int w = threadIdx.x >> 5, ln = threadIdx.x & 31;
  float mx = a.m.sink ? a.m.sink[h] : -INFINITY, l = a.m.sink ? 1.f : 0.f;
  __syncthreads();
  for (int t = k0 / PAGE_TOKENS; t <= pos / PAGE_TOKENS; ++t) {
    const int page = a.block_table[(int64_t)lane * a.max_pages + t];
    const T* base = reinterpret_cast<const T*>(a.cache) + (int64_t)page * PAGE_TOKENS * a.ldc;
    for (int j = w; j < PAGE_TOKENS; j += 4) {
      const int key = t * PAGE_TOKENS + j;
      float s = 0.f;
      if (key >= k0 && key <= pos)
        for (int i = ln; i < dt; i += 32) s = fmaf(q[i], ldf<T>(base[(int64_t)j * a.ldc + i]), s);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      if (ln == 0) sc[j] = (key >= k0 && key <= pos) ? s * a.m.scale : -INFINITY;
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
    const int j0 = max(0, k0 - t * PAGE_TOKENS), j1 = min(PAGE_TOKENS - 1, pos - t * PAGE_TOKENS);
    for (int i = threadIdx.x; i < r; i += 128) {
      float v = acc[i] * alpha;
      for (int j = j0; j <= j1; ++j) v = fmaf(sc[j], ldf<T>(base[(int64_t)j * a.ldc + i]), v);
      acc[i] = v;
    }
    __syncthreads();
  }
  const int64_t o = (row * a.m.heads + h) * a.kv_splits;
  for (int i = threadIdx.x; i < r; i += 128) a.olat[o * r + i] = acc[i];
  if (threadIdx.x == 0) a.ml[o] = make_float2(mx, l);
}

// out[row][head] = gate * W_uv (o_lat / l)
template <typename T>
__global__ void __launch_bounds__(128) latent_out_plain_kernel(LatentAttnArgs a) {
  extern __shared__ float so[];
  pdl_launch_dependents();
  pdl_wait();
  int64_t row;
  if (!tile_row(a.tiles, a.max_tile_rows, row)) return;
  const int h = blockIdx.y, r = a.m.kv_rank, dv = a.m.vdim;
  const int64_t o = (row * a.m.heads + h) * a.kv_splits;
  const float inv = 1.0f / a.ml[o].y;
  for (int i = threadIdx.x; i < r; i += 128) so[i] = ldf<T>(stf<T>(a.olat[o * r + i] * inv));
  __syncthreads();
  const float g = a.m.gate ? a.gate[row * a.m.heads + h] : 1.0f;
  const T* w = reinterpret_cast<const T*>(a.ukv) + (int64_t)a.m.heads * a.m.dim + (int64_t)h * dv;
  T* op = reinterpret_cast<T*>(a.out) + row * a.ldo + (int64_t)h * dv;
  for (int j = threadIdx.x; j < dv; j += 128) {
    float acc = 0.f;
    for (int i = 0; i < r; ++i) acc = fmaf(so[i], ldf<T>(w[(int64_t)i * a.ld_ukv + j]), acc);
    op[j] = stf<T>(acc * g);
  }
}

// ------------------------------------------------------------------ bf16 kernels on the tensor cores
// Three launches per layer: queries into the latent space, attention over the cache rows, values back out of it.

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_all;" ::: "memory"); }

// rows x cols (bf16, row stride lds elements) -> shared memory with row stride ldd elements; columns up to cols_p
// and rows up to rows_p are zero-filled.  Asynchronous where 16-byte copies are possible.
__device__ __forceinline__ void stage_matrix(bf16* dst, int ldd, const bf16* src, int64_t lds, int rows, int cols, int rows_p, int cols_p,
                                             bool vec) {
  const int cpr = cols_p / 8;
  for (int i = threadIdx.x; i < rows_p * cpr; i += blockDim.x) {
    const int r = i / cpr, c = (i % cpr) * 8;
    bf16* d = dst + (int64_t)r * ldd + c;
    if (r < rows && c + 8 <= cols && vec) {
      cp_async16(smem_u32(d), src + r * lds + c);
    } else {
#pragma unroll
      for (int e = 0; e < 8; ++e) d[e] = (r < rows && c + e < cols) ? src[r * lds + c + e] : __float2bfloat16_rn(0.f);
    }
  }
}

__device__ __forceinline__ int2 chunk_rows(const LatentAttnArgs& a, int i) {
  if (a.chunks.list) return a.chunks.list[i];
  const int r0 = i * kChunkRows;
  return make_int2(r0, (int)min((int64_t)kChunkRows, a.rows - r0));
}

// Two neighbouring query values of a row (col even) from the projection's slabs or its bf16 output.
__device__ __forceinline__ float2 q_pair(const LatentAttnArgs& a, int64_t row, int64_t col) {
  if (a.nsplit == 0) {
    const __nv_bfloat162 v = *reinterpret_cast<const __nv_bfloat162*>(reinterpret_cast<const bf16*>(a.q) + row * a.ldq + col);
    return make_float2(__low2float(v), __high2float(v));
  }
  float2 t = make_float2(0.f, 0.f);
  const float* p = reinterpret_cast<const float*>(a.q) + row * a.ldq + col;
  for (int s = 0; s < a.nsplit; ++s) {
    const float2 v = *reinterpret_cast<const float2*>(p + s * a.split_stride);
    t.x += v.x;
    t.y += v.y;
  }
  return t;
}

constexpr int LQ_N = 64;   // latent features per CTA

// grid (latent tiles, heads, chunks): qeff[row][head][n0 .. n0+63] = sum_i q[row][head][i] W_uk[n][i]; the
// head's rot_dim part is rotated on the way.
__global__ void __launch_bounds__(256) latent_q_kernel(LatentAttnArgs a) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  const int h = blockIdx.y, dn = a.m.dim, dr = a.m.rot_dim, r = a.m.kv_rank;
  const int kp = (dn + 15) / 16 * 16, ld = kp + 8;
  bf16* sA = reinterpret_cast<bf16*>(smem_raw);
  bf16* sB = sA + kChunkRows * ld;
  const int n0 = blockIdx.x * LQ_N;
  pdl_launch_dependents();
  // the weights do not depend on earlier kernels
  stage_matrix(sB, ld, reinterpret_cast<const bf16*>(a.ukv) + (int64_t)n0 * a.ld_ukv + (int64_t)h * dn, a.ld_ukv, min(LQ_N, r - n0), dn, LQ_N, kp,
               dn % 8 == 0);
  pdl_wait();
  const int2 ch = chunk_rows(a, blockIdx.z);
  const int64_t qcol = (int64_t)h * (dn + dr);
  const bool even = (dn % 2 == 0) && (dr % 2 == 0);
  const int rows16 = (ch.y + 15) / 16 * 16;
  if (a.nsplit > 0 && dn % 4 == 0 && qcol % 4 == 0) {
    // four columns a thread, four independent chains of slab loads in flight
    const int hp = kp / 4, items = rows16 * hp;
    for (int i0 = threadIdx.x; i0 < items; i0 += 4 * 256) {
      float4 v[4];
      const float* src[4];
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int i = i0 + u * 256, row = i / hp, c = (i % hp) * 4;
        src[u] = i < items && row < ch.y && c < dn ? reinterpret_cast<const float*>(a.q) + (int64_t)(ch.x + row) * a.ldq + qcol + c : nullptr;
        v[u] = make_float4(0.f, 0.f, 0.f, 0.f);
      }
      for (int s = 0; s < a.nsplit; ++s)
#pragma unroll
        for (int u = 0; u < 4; ++u)
          if (src[u]) add4(v[u], *reinterpret_cast<const float4*>(src[u] + s * a.split_stride));
#pragma unroll
      for (int u = 0; u < 4; ++u) {
        const int i = i0 + u * 256;
        if (i < items) *reinterpret_cast<uint2*>(sA + (i / hp) * ld + (i % hp) * 4) = make_uint2(pack_bf16(v[u].x, v[u].y), pack_bf16(v[u].z, v[u].w));
      }
    }
  } else {
    const int hp = kp / 2;
    for (int i = threadIdx.x; i < rows16 * hp; i += 256) {
      const int row = i / hp, c = (i % hp) * 2;
      float2 v = make_float2(0.f, 0.f);
      if (row < ch.y && c < dn) {
        if (even) v = q_pair(a, ch.x + row, qcol + c);
        else {
          v.x = q_at<bf16>(a, ch.x + row, qcol + c);
          if (c + 1 < dn) v.y = q_at<bf16>(a, ch.x + row, qcol + c + 1);
        }
      }
      *reinterpret_cast<uint32_t*>(sA + row * ld + c) = pack_bf16(v.x, v.y);
    }
  }
  {
    const int half = a.m.rope_dims / 2, np = (dr + 1) / 2;   // the rotations are shared out over the latent tiles
    for (int i = blockIdx.x * 256 + threadIdx.x; i < ch.y * np; i += gridDim.x * 256) {
      const int64_t row = ch.x + i / np;
      const int p = i % np;
      float2 v;
      if (even) v = q_pair(a, row, qcol + dn + 2 * p);
      else v = make_float2(q_at<bf16>(a, row, qcol + dn + 2 * p), 2 * p + 1 < dr ? q_at<bf16>(a, row, qcol + dn + 2 * p + 1) : 0.f);
      v = make_float2(ldf<bf16>(stf<bf16>(v.x)), ldf<bf16>(stf<bf16>(v.y)));   // the projection's bf16 output
      if (p < half) {
        const int pos = min(max(row_pos(a.map, row), 0), a.m.max_pos - 1);
        v = rotate(v, a.m.rope[(int64_t)pos * half + p]);
      }
      bf16* qe = reinterpret_cast<bf16*>(a.qeff) + (row * a.m.heads + h) * a.ldc + r + 2 * p;
      qe[0] = stf<bf16>(v.x);
      if (2 * p + 1 < dr) qe[1] = stf<bf16>(v.y);
    }
  }
  cp_async_wait();
  __syncthreads();
  // warps: wm along the rows (16 each), the others along the 64 latent features
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, l8 = lane & 7, lq = lane >> 3, g = lane >> 2, t = lane & 3;
  const int wm = ch.y <= 16 ? 1 : ch.y <= 32 ? 2 : 4, wn = 4 / wm, nt_n = 8 / wn;
  const int mrow = (warp % wm) * 16, ncol = (warp / wm) * nt_n * 8;
  if (warp >= 4 || mrow >= rows16) return;
  float acc[8][4];
#pragma unroll
  for (int i = 0; i < 8; ++i)
#pragma unroll
    for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
  const uint32_t aA = smem_u32(sA), aB = smem_u32(sB);
  for (int k = 0; k < kp; k += 16) {
    uint32_t af[4];
    ldmatrix_x4(af[0], af[1], af[2], af[3], aA + ((mrow + (lq & 1) * 8 + l8) * ld + k + (lq >> 1) * 8) * 2);
#pragma unroll
    for (int i = 0; i < 8; i += 2) {
      if (i >= nt_n) break;
      uint32_t b0, b1, b2, b3;
      ldmatrix_x4(b0, b1, b2, b3, aB + ((ncol + i * 8 + (lq >> 1) * 8 + l8) * ld + k + (lq & 1) * 8) * 2);
      mma_bf16_16816(acc[i], af, b0, b1);
      mma_bf16_16816(acc[i + 1], af, b2, b3);
    }
  }
#pragma unroll
  for (int i = 0; i < 8; ++i) {
    if (i >= nt_n) break;
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int row = mrow + g + hf * 8, n = n0 + ncol + i * 8 + 2 * t;
      if (row >= ch.y || n >= r) continue;
      bf16* qe = reinterpret_cast<bf16*>(a.qeff) + ((int64_t)(ch.x + row) * a.m.heads + h) * a.ldc + n;
      if (n + 1 < r && (r & 1) == 0) *reinterpret_cast<uint32_t*>(qe) = pack_bf16(acc[i][2 * hf], acc[i][2 * hf + 1]);
      else {
        qe[0] = stf<bf16>(acc[i][2 * hf]);
        if (n + 1 < r) qe[1] = stf<bf16>(acc[i][2 * hf + 1]);
      }
    }
  }
}

// Attention of a few (token, head) rows over the cache rows of their lane.  grid (kv splits, tiles * subtiles, head
// groups), 256 threads.  A CTA's 16 * MT rows are `heads_per` heads of up to `tokens_per` tokens.  Per 64-key page:
//   S     warp w: keys 16 (w & 3) .. +15, half (w >> 2) of the features; the halves meet in shared memory
//   P     online softmax in f32, 16 / MT threads per row
//   O     warp w: value columns 16 (w + 8 i) .. +15, f32 in registers
// The page's [64][kv_rank + rot_dim] rows are both keys and (their first kv_rank columns) values: one TMA load each.
struct AbsCfg {
  int boxes;       // 64-column boxes of a cache row
  int stages;
  int heads_per, tokens_per, subtiles;
};
constexpr int ABS_OG = 4;       // 16-column value groups per warp: kv_rank up to 512

template <int MT>
__global__ void __launch_bounds__(288) latent_attn_kernel(const __grid_constant__ CUtensorMap tm, LatentAttnArgs a, AbsCfg cf) {
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  constexpr int R = 16 * MT, TPR = 256 / R, KPT = 64 / TPR;   // rows, threads per row, keys per thread
  const int stage_bytes = cf.boxes * 8192;
  uint8_t* sKV = smem;
  uint8_t* sQ = sKV + cf.stages * stage_bytes;                // [box][R rows][128 bytes]
  uint8_t* sP = sQ + cf.boxes * R * 128;                      // [R rows][128 bytes]
  float* sS = reinterpret_cast<float*>(sP + R * 128);         // [2][R][68]
  float* sAl = sS + 2 * R * 68;                               // [R]
  uint64_t* full = reinterpret_cast<uint64_t*>(sAl + R);      // [stages] filled by TMA
  uint64_t* empty = full + 4;                                 // [stages] released by the eight consumer warps
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, l8 = lane & 7, lq = lane >> 3, g = lane >> 2, t = lane & 3;
  if (tid == 256) {
    for (int i = 0; i < cf.stages; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 8);
    }
    fence_barrier_init();
    tma_prefetch_desc(&tm);
  }
  pdl_launch_dependents();
  __syncthreads();
  // In a captured decode step positions and block tables predate the step, and so do all cache rows but the newest.
  if (!a.early_kv) pdl_wait();
  const int2 tr = tile_rows(a.tiles, (int)blockIdx.y / cf.subtiles);
  const int tok0 = ((int)blockIdx.y % cf.subtiles) * cf.tokens_per;
  const int ntok = min(cf.tokens_per, tr.y - tok0);
  if (ntok <= 0) return;
  const int64_t row0 = tr.x + tok0;
  const int head0 = blockIdx.z * cf.heads_per, nh = min(cf.heads_per, a.m.heads - head0);
  const int lane_id = row_lane(a.map, row0);
  const int cap = a.max_pages * PAGE_TOKENS;
  const int pos_first = min(max(row_pos(a.map, row0), 0), cap - 1), pos_last = min(pos_first + ntok - 1, cap - 1);
  const int k_lo = a.m.window > 0 ? max(0, pos_first - a.m.window + 1) : 0;
  const int t_lo = k_lo / PAGE_TOKENS, nt_all = pos_last / PAGE_TOKENS - t_lo + 1;
  const int per = (nt_all + (int)gridDim.x - 1) / (int)gridDim.x;
  const int t0 = t_lo + (int)blockIdx.x * per, nt = max(0, min(per, t_lo + nt_all - t0));
  if (warp == 8) {
    // ---- producer
    if (lane == 0) {
      auto load_page = [&](int i) {
        const int st = i % cf.stages;
        const int page = a.block_table[(int64_t)lane_id * a.max_pages + t0 + i];
        mbar_expect_tx(&full[st], stage_bytes);
        for (int b = 0; b < cf.boxes; ++b) tma_load_2d(sKV + st * stage_bytes + b * 8192, &tm, &full[st], b * 64, page * PAGE_TOKENS);
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
  // queries
  for (int i = tid; i < R * cf.boxes * 8; i += 256) {
    const int m = i / (cf.boxes * 8), c = i % (cf.boxes * 8);
    const int tok = m / cf.heads_per, hh = m % cf.heads_per;
    uint4 v = make_uint4(0, 0, 0, 0);
    if (tok < ntok && hh < nh && c * 8 < a.ldc)
      v = *reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(a.qeff) + ((row0 + tok) * a.m.heads + head0 + hh) * a.ldc + c * 8);
    *reinterpret_cast<uint4*>(sQ + (c >> 3) * (R * 128) + swz128((uint32_t)m, (uint32_t)(c & 7))) = v;
  }
  auto consumers_sync = [] { asm volatile("bar.sync 1, 256;" ::: "memory"); };
  consumers_sync();

  // softmax ownership: thread -> (row, KPT keys)
  const int srow = tid / TPR, skey = (tid % TPR) * KPT;
  const int stok = srow / cf.heads_per;
  const bool sval = stok < ntok && srow % cf.heads_per < nh;
  const int spos = pos_first + stok, slo = a.m.window > 0 ? spos - a.m.window : -1;   // sees keys slo < key <= spos
  float m_run = -INFINITY, l_run = 0.f;
  float acc[MT][ABS_OG][2][4];
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int j = 0; j < ABS_OG; ++j)
#pragma unroll
      for (int e = 0; e < 8; ++e) acc[i][j][e >> 2][e & 3] = 0.f;
  const int groups = (a.m.kv_rank + 15) / 16;
  const int kg = warp & 3, kh = warp >> 2;
  // Lane addresses.  Every row an ldmatrix lane points at is l8 modulo 8, so the swizzle is a constant of the lane and
  // the loops below add constants only.  Half kh of the features: 16-feature steps 2 kh and 2 kh + 1 of every box.
  uint32_t k_off[2], q_off[2], p_off[4];
#pragma unroll
  for (int u = 0; u < 2; ++u) {
    const uint32_t ch = (2 * kh + u) * 2;
    k_off[u] = swz128(kg * 16 + (lq >> 1) * 8 + l8, ch + (lq & 1));
    q_off[u] = smem_u32(sQ) + swz128((lq & 1) * 8 + l8, ch + (lq >> 1));
  }
#pragma unroll
  for (int k = 0; k < 4; ++k) p_off[k] = smem_u32(sP) + swz128((lq & 1) * 8 + l8, k * 2 + (lq >> 1));
  const uint32_t v_off = (warp >> 2) * 8192 + swz128((lq & 1) * 8 + l8, (warp & 3) * 2 + (lq >> 1));
  const uint32_t kv_base = smem_u32(sKV);
  float* const s_row = sS + (kh * R + g) * 68 + kg * 16 + 2 * t;
  bool ok = true;
  for (int it = 0; it < nt; ++it) {
    const int st = it % cf.stages;
    if (ok) ok = mbar_wait(&full[st], (it / cf.stages) & 1, a.status);
    const uint32_t kv = kv_base + st * stage_bytes;
    float sc[MT][2][4];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int e = 0; e < 8; ++e) sc[i][e >> 2][e & 3] = 0.f;
    // the fragments of the next box are requested ahead of this box's products
    uint32_t bf[2][2][4], af[2][2][MT][4];
    auto fetch = [&](int slot, uint32_t kb, uint32_t qb) {
#pragma unroll
      for (int u = 0; u < 2; ++u) {
        ldmatrix_x4(bf[slot][u][0], bf[slot][u][1], bf[slot][u][2], bf[slot][u][3], kb + k_off[u]);
#pragma unroll
        for (int i = 0; i < MT; ++i)
          ldmatrix_x4(af[slot][u][i][0], af[slot][u][i][1], af[slot][u][i][2], af[slot][u][i][3], qb + q_off[u] + i * 2048);
      }
    };
    auto products = [&](int slot) {
#pragma unroll
      for (int u = 0; u < 2; ++u)
#pragma unroll
        for (int i = 0; i < MT; ++i) {
          mma_bf16_16816(sc[i][0], af[slot][u][i], bf[slot][u][0], bf[slot][u][1]);
          mma_bf16_16816(sc[i][1], af[slot][u][i], bf[slot][u][2], bf[slot][u][3]);
        }
    };
    fetch(0, kv, 0);
    for (int b = 0; b < cf.boxes; b += 2) {
      if (b + 1 < cf.boxes) fetch(1, kv + (b + 1) * 8192, (b + 1) * (R * 128));
      products(0);
      if (b + 1 >= cf.boxes) break;
      if (b + 2 < cf.boxes) fetch(0, kv + (b + 2) * 8192, (b + 2) * (R * 128));
      products(1);
    }
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int hf = 0; hf < 2; ++hf)
          *reinterpret_cast<float2*>(s_row + (i * 16 + hf * 8) * 68 + n * 8) = make_float2(sc[i][n][2 * hf], sc[i][n][2 * hf + 1]);
    consumers_sync();
    {
      const int key0 = (t0 + it) * PAGE_TOKENS + skey;
      float x[KPT], mx = -INFINITY;
#pragma unroll
      for (int e = 0; e < KPT; e += 4) {
        const float4 s0 = *reinterpret_cast<const float4*>(sS + srow * 68 + skey + e), s1 = *reinterpret_cast<const float4*>(sS + (R + srow) * 68 + skey + e);
        x[e] = s0.x + s1.x;
        x[e + 1] = s0.y + s1.y;
        x[e + 2] = s0.z + s1.z;
        x[e + 3] = s0.w + s1.w;
      }
#pragma unroll
      for (int e = 0; e < KPT; ++e) {
        x[e] = (sval && key0 + e <= spos && key0 + e > slo) ? x[e] * a.m.scale : -INFINITY;
        mx = fmaxf(mx, x[e]);
      }
#pragma unroll
      for (int o = TPR / 2; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
      const float m_new = fmaxf(m_run, mx), m_use = m_new == -INFINITY ? 0.f : m_new;
      const float alpha = __expf(m_run - m_use);
      uint32_t pk[KPT / 2];
      float ps = 0.f;
#pragma unroll
      for (int e = 0; e < KPT; e += 2) {
        const float p0 = __expf(x[e] - m_use), p1 = __expf(x[e + 1] - m_use);
        ps += p0 + p1;
        pk[e / 2] = pack_bf16(p0, p1);
      }
      l_run = l_run * alpha + ps;   // this thread's keys; the row's threads meet after the last page
      m_run = m_new;
      uint8_t* pd = sP + swz128((uint32_t)srow, (uint32_t)(skey >> 3)) + (skey & 7) * 2;
#pragma unroll
      for (int e = 0; e < KPT / 2; ++e) *reinterpret_cast<uint32_t*>(pd + e * 4) = pk[e];
      if (tid % TPR == 0) sAl[srow] = alpha;
    }
    consumers_sync();
#pragma unroll
    for (int i = 0; i < MT; ++i) {
      const float a0 = sAl[i * 16 + g], a1 = sAl[i * 16 + g + 8];
      if (__any_sync(0xffffffffu, a0 != 1.f || a1 != 1.f)) {
#pragma unroll
        for (int j = 0; j < ABS_OG; ++j)
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            acc[i][j][n][0] *= a0;
            acc[i][j][n][1] *= a0;
            acc[i][j][n][2] *= a1;
            acc[i][j][n][3] *= a1;
          }
      }
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) {   // 16 keys a step
      uint32_t pf[MT][4], vf[ABS_OG][4];
#pragma unroll
      for (int i = 0; i < MT; ++i) ldmatrix_x4(pf[i][0], pf[i][1], pf[i][2], pf[i][3], p_off[k] + i * 2048);
#pragma unroll
      for (int j = 0; j < ABS_OG; ++j)   // value columns 16 (warp + 8 j) ..: box (warp >> 2) + 2 j
        if (warp + 8 * j < groups) ldmatrix_x4_trans(vf[j][0], vf[j][1], vf[j][2], vf[j][3], kv + v_off + j * 16384 + k * 2048);
#pragma unroll
      for (int j = 0; j < ABS_OG; ++j) {
        if (warp + 8 * j >= groups) break;
#pragma unroll
        for (int i = 0; i < MT; ++i) {
          mma_bf16_16816(acc[i][j][0], pf[i], vf[j][0], vf[j][1]);
          mma_bf16_16816(acc[i][j][1], pf[i], vf[j][2], vf[j][3]);
        }
      }
    }
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[st]);
    // the next scores go to a buffer every warp has left: the probabilities and factors are rewritten only behind
    // the next barrier, which every warp reaches after this page's products
  }
#pragma unroll
  for (int o = TPR / 2; o > 0; o >>= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, o);
  if (!ok) return;
#pragma unroll
  for (int i = 0; i < MT; ++i)
#pragma unroll
    for (int hf = 0; hf < 2; ++hf) {
      const int m = i * 16 + g + hf * 8, tok = m / cf.heads_per, hh = m % cf.heads_per;
      if (tok >= ntok || hh >= nh) continue;
      const int64_t u = ((row0 + tok) * a.m.heads + head0 + hh) * a.kv_splits + blockIdx.x;
      float* o = a.olat + u * a.m.kv_rank;
#pragma unroll
      for (int j = 0; j < ABS_OG; ++j)
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          const int col = (warp + 8 * j) * 16 + n * 8 + 2 * t;
          if (col + 1 < a.m.kv_rank && (a.m.kv_rank & 1) == 0)
            *reinterpret_cast<float2*>(o + col) = make_float2(acc[i][j][n][2 * hf], acc[i][j][n][2 * hf + 1]);
          else {
            if (col < a.m.kv_rank) o[col] = acc[i][j][n][2 * hf];
            if (col + 1 < a.m.kv_rank) o[col + 1] = acc[i][j][n][2 * hf + 1];
          }
        }
    }
  if (tid % TPR == 0 && sval)
    a.ml[((row0 + stok) * a.m.heads + head0 + srow % cf.heads_per) * a.kv_splits + blockIdx.x] = make_float2(m_run, l_run);
}

constexpr int LO_ROWS = 16, LO_N = 32, LO_PARTS = kChunkRows / LO_ROWS;

// grid (value tiles, heads, chunks * LO_PARTS), 256 threads: merges the kv splits, then
// out[row][head][n0 .. n0+31] = gate * sum_k o[k] W_uv[k][n].  Warp w: columns 8 (w & 3) .. +7, half (w >> 2) of k.
__global__ void __launch_bounds__(256) latent_out_kernel(LatentAttnArgs a) {
  extern __shared__ __align__(16) uint8_t smem_raw[];
  const int h = blockIdx.y, r = a.m.kv_rank, dv = a.m.vdim;
  const int kp = (r + 63) / 64 * 64, ld = kp + 8;   // two halves of whole 32-wide steps
  bf16* sA = reinterpret_cast<bf16*>(smem_raw);
  bf16* sB = sA + LO_ROWS * ld;                 // [kp][LO_N + 8]
  constexpr int ldb = LO_N + 8;
  __shared__ float sw[LO_ROWS][17];
  __shared__ float sred[4][32][4];
  const int n0 = blockIdx.x * LO_N, tid = threadIdx.x;
  pdl_launch_dependents();
  if (!a.chunks.list && (int64_t)blockIdx.z * LO_ROWS >= a.rows) return;   // a uniform step knows its rows without loading anything
  const int64_t c0 = (int64_t)a.m.heads * a.m.dim + (int64_t)h * dv + n0;
  stage_matrix(sB, ldb, reinterpret_cast<const bf16*>(a.ukv) + c0, a.ld_ukv, r, min(LO_N, dv - n0), kp, LO_N, c0 % 8 == 0);
  pdl_wait();
  int2 ch = chunk_rows(a, (int)blockIdx.z / LO_PARTS);
  const int skip = ((int)blockIdx.z % LO_PARTS) * LO_ROWS;
  ch.x += skip;
  ch.y = min(LO_ROWS, ch.y - skip);
  if (ch.y <= 0) {
    cp_async_wait();
    return;
  }
  const int ns = a.kv_splits;
  {
    // weights of the splits, exp(m_s - M) / sum: 16 threads a row, one split each
    const int row = tid >> 4, s = tid & 15;
    const bool in = row < ch.y && s < ns;
    const float2 ml = in ? a.ml[((int64_t)(ch.x + row) * a.m.heads + h) * ns + s] : make_float2(-INFINITY, 0.f);
    const float sink = a.m.sink ? a.m.sink[h] : -INFINITY;
    float M = fmaxf(ml.x, sink);
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
    const float f = ml.x == -INFINITY ? 0.f : __expf(ml.x - M);
    float L = ml.y * f;
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) L += __shfl_xor_sync(0xffffffffu, L, o);
    if (a.m.sink) L += __expf(sink - M);
    sw[row][s] = L > 0.f ? f / L : 0.f;
  }
  __syncthreads();
  if (r % 4 == 0) {
    // four columns a thread, eight independent chains of split loads in flight
    constexpr int U = 8;
    const int hp = kp / 4, items = LO_ROWS * hp;
    for (int i0 = tid; i0 < items; i0 += U * 256) {
      float4 v[U];
      const float* src[U];
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int i = i0 + u * 256, row = i / hp, c = (i % hp) * 4;
        src[u] = row < ch.y && c < r ? a.olat + ((int64_t)(ch.x + row) * a.m.heads + h) * ns * r + c : nullptr;
        v[u] = make_float4(0.f, 0.f, 0.f, 0.f);
      }
#pragma unroll 2
      for (int s = 0; s < ns; ++s) {
        float4 x[U];
#pragma unroll
        for (int u = 0; u < U; ++u) x[u] = src[u] ? *reinterpret_cast<const float4*>(src[u] + (int64_t)s * r) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int u = 0; u < U; ++u) {
          const float f = sw[min((i0 + u * 256) / hp, LO_ROWS - 1)][s];
          v[u].x = fmaf(f, x[u].x, v[u].x);
          v[u].y = fmaf(f, x[u].y, v[u].y);
          v[u].z = fmaf(f, x[u].z, v[u].z);
          v[u].w = fmaf(f, x[u].w, v[u].w);
        }
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const int i = i0 + u * 256;
        if (i < items) *reinterpret_cast<uint2*>(sA + (i / hp) * ld + (i % hp) * 4) = make_uint2(pack_bf16(v[u].x, v[u].y), pack_bf16(v[u].z, v[u].w));
      }
    }
  } else {
    for (int i = tid; i < LO_ROWS * kp; i += 256) {
      const int row = i / kp, c = i % kp;
      float v = 0.f;
      if (row < ch.y && c < r)
        for (int s = 0; s < ns; ++s) v += sw[row][s] * a.olat[(((int64_t)(ch.x + row) * a.m.heads + h) * ns + s) * r + c];
      sA[row * ld + c] = stf<bf16>(v);
    }
  }
  cp_async_wait();
  __syncthreads();
  const int warp = tid >> 5, lane = tid & 31, l8 = lane & 7, lq = lane >> 3, g = lane >> 2, t = lane & 3;
  const int nq = warp & 3, kh = warp >> 2;
  float acc[4] = {};
  const uint32_t aA = smem_u32(sA), aB = smem_u32(sB);
  for (int k = kh * (kp / 2); k < (kh + 1) * (kp / 2); k += 32) {
    uint32_t a0[4], a1[4], b0, b1, b2, b3;
    ldmatrix_x4(a0[0], a0[1], a0[2], a0[3], aA + (((lq & 1) * 8 + l8) * ld + k + (lq >> 1) * 8) * 2);
    ldmatrix_x4(a1[0], a1[1], a1[2], a1[3], aA + (((lq & 1) * 8 + l8) * ld + k + 16 + (lq >> 1) * 8) * 2);
    ldmatrix_x4_trans(b0, b1, b2, b3, aB + ((k + lq * 8 + l8) * ldb + nq * 8) * 2);
    mma_bf16_16816(acc, a0, b0, b1);
    mma_bf16_16816(acc, a1, b2, b3);
  }
  if (kh == 1) *reinterpret_cast<float4*>(sred[nq][lane]) = make_float4(acc[0], acc[1], acc[2], acc[3]);
  __syncthreads();
  if (kh == 1) return;
#pragma unroll
  for (int hf = 0; hf < 2; ++hf) {
    const int row = g + hf * 8, n = n0 + nq * 8 + 2 * t;
    if (row >= ch.y || n >= dv) continue;
    const float gt = a.m.gate ? a.gate[(int64_t)(ch.x + row) * a.m.heads + h] : 1.0f;
    bf16* op = reinterpret_cast<bf16*>(a.out) + (int64_t)(ch.x + row) * a.ldo + (int64_t)h * dv + n;
    op[0] = stf<bf16>((acc[2 * hf] + sred[nq][lane][2 * hf]) * gt);
    if (n + 1 < dv) op[1] = stf<bf16>((acc[2 * hf + 1] + sred[nq][lane][2 * hf + 1]) * gt);
  }
}

template <typename T>
__global__ void __launch_bounds__(128) gather_rows_kernel(const T* src, const int* index, T* dst, int64_t width) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t from = index[blockIdx.x];
  for (int64_t i = threadIdx.x; i < width; i += 128) dst[blockIdx.x * width + i] = src[from * width + i];
}

template <typename T>
int plain_launch(Ctx* c, const LatentAttnArgs& a) {
  const dim3 grid((unsigned)(a.tiles.count * a.max_tile_rows), (unsigned)a.m.heads);
  const int dt = a.m.kv_rank + a.m.rot_dim;
  const size_t s1 = (size_t)(a.m.dim + a.m.rot_dim) * 4, s2 = (size_t)(dt + a.m.kv_rank + PAGE_TOKENS) * 4, s3 = (size_t)a.m.kv_rank * 4;
  RB_REQUIRE(s1 <= 48 * 1024 && s2 <= 48 * 1024, "latent attention: head or latent size too large");
  RB_CUDA(launch_k(latent_q_plain_kernel<T>, grid, dim3(128), s1, c->stream, c->use_pdl, a));
  RB_CUDA(launch_k(latent_attn_plain_kernel<T>, grid, dim3(128), s2, c->stream, c->use_pdl, a));
  RB_CUDA(launch_k(latent_out_plain_kernel<T>, grid, dim3(128), s3, c->stream, c->use_pdl, a));
  g_launch_total += 3;
  return REWB200_OK;
}

}  // namespace

int latent_post_launch(Ctx* c, const LatentPostArgs& a, int64_t rows) {
  if (rows == 0) return REWB200_OK;
  const size_t smem = (size_t)a.ld * sizeof(float);
  RB_REQUIRE(a.ld % 4 == 0 && smem <= 48 * 1024, "latent attention: the input projection is wider than 12288 columns");
  const bool small = rows <= 256;
  const int nv = (int)((a.ld + 127) / 128);
  if (rows >= 1024 && nv <= 20 && a.m.q_rank % 4 == 0 && a.m.kv_rank % 4 == 0 && a.m.rot_dim % 4 == 0) {
    auto go = [&](auto kernel) { return launch_k(kernel, dim3((unsigned)((rows + 7) / 8)), dim3(256), 0, c->stream, c->use_pdl, a, rows); };
#define RB_LPOST(T) (nv <= 5 ? go(latent_post_rows_kernel<T, 5>) : nv <= 10 ? go(latent_post_rows_kernel<T, 10>) : nv <= 16 ? go(latent_post_rows_kernel<T, 16>) : go(latent_post_rows_kernel<T, 20>))
    RB_CUDA(a.dtype == REWB200_BF16 ? RB_LPOST(bf16) : RB_LPOST(float));
#undef RB_LPOST
    ++g_launch_total;
    return REWB200_OK;
  }
  const dim3 grid((unsigned)rows), block(small ? (unsigned)std::min<int64_t>(768, std::max<int64_t>(64, (a.ld / 4 + 31) / 32 * 32)) : 128);
  cudaError_t e;
  if (a.dtype == REWB200_BF16)
    e = small ? launch_k(latent_post_kernel<bf16, true>, grid, block, smem, c->stream, c->use_pdl, a)
              : launch_k(latent_post_kernel<bf16, false>, grid, block, smem, c->stream, c->use_pdl, a);
  else
    e = small ? launch_k(latent_post_kernel<float, true>, grid, block, smem, c->stream, c->use_pdl, a)
              : launch_k(latent_post_kernel<float, false>, grid, block, smem, c->stream, c->use_pdl, a);
  RB_CUDA(e);
  ++g_launch_total;
  return REWB200_OK;
}

namespace {

constexpr size_t kSmemMax = 227 * 1024;

// Sizes the tensor-core kernels take; everything else runs on the plain ones.
bool abs_config(const LatentDims& m, int64_t ldc, int mt, AbsCfg* cf, size_t* smem) {
  cf->boxes = (int)((m.kv_rank + m.rot_dim + 63) / 64);
  const int R = 16 * mt;
  const size_t fixed = (size_t)cf->boxes * R * 128 + R * 128 + 2 * R * 68 * 4 + R * 4 + 128 + 1024;
  cf->stages = 4;
  while (cf->stages > 1 && fixed + (size_t)cf->stages * cf->boxes * 8192 > kSmemMax) --cf->stages;
  *smem = fixed + (size_t)cf->stages * cf->boxes * 8192;
  const size_t q_smem = (size_t)2 * 64 * ((m.dim + 15) / 16 * 16 + 8) * 2;
  const int kp = (m.kv_rank + 63) / 64 * 64;
  const size_t o_smem = (size_t)LO_ROWS * (kp + 8) * 2 + (size_t)kp * (LO_N + 8) * 2;
  (void)ldc;
  return m.kv_rank <= 16 * 8 * ABS_OG && *smem <= kSmemMax && cf->stages >= 2 && q_smem <= kSmemMax && o_smem <= kSmemMax - 8192;
}

}  // namespace

int latent_kv_splits(Ctx* c, const LatentDims& m, int64_t tiles, int64_t max_ctx) {
  const int64_t ctx = m.window > 0 ? std::min<int64_t>(m.window, max_ctx) : max_ctx;
  const int64_t pages = (ctx + PAGE_TOKENS - 1) / PAGE_TOKENS + 1;
  const int64_t hg = (m.heads + 31) / 32;
  const int64_t want = c->sm_count / std::max<int64_t>(1, tiles * hg);
  return (int)std::max<int64_t>(1, std::min<int64_t>(std::min<int64_t>(want, pages), 8));
}

int latent_attn_absorbed_launch(Ctx* c, const LatentAttnArgs& a) {
  if (a.tiles.count == 0) return REWB200_OK;
  AbsCfg cf;
  size_t smem = 0;
  const int mt = a.m.heads <= 16 && a.max_tile_rows == 1 ? 1 : 2;
  if (a.dtype != REWB200_BF16 || c->latent_impl == 1 || !abs_config(a.m, a.ldc, mt, &cf, &smem)) {
    // the plain kernels do not split the keys: one partial per (row, head)
    LatentAttnArgs p = a;
    p.kv_splits = 1;
    return a.dtype == REWB200_BF16 ? plain_launch<bf16>(c, p) : plain_launch<float>(c, p);
  }
  cf.heads_per = std::min(a.m.heads, 16 * mt);
  cf.tokens_per = std::min(16 * mt / cf.heads_per, a.max_tile_rows);
  cf.subtiles = (a.max_tile_rows + cf.tokens_per - 1) / cf.tokens_per;
  const int kp = (a.m.dim + 15) / 16 * 16, rp = (a.m.kv_rank + 63) / 64 * 64;
  const size_t q_smem = (size_t)(kChunkRows + LQ_N) * (kp + 8) * 2;
  const size_t o_smem = (size_t)LO_ROWS * (rp + 8) * 2 + (size_t)rp * (LO_N + 8) * 2;
  static bool attr_set = false;
  if (!attr_set) {
    RB_CUDA(cudaFuncSetAttribute(latent_q_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemMax));
    RB_CUDA(cudaFuncSetAttribute(latent_attn_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemMax));
    RB_CUDA(cudaFuncSetAttribute(latent_attn_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemMax));
    RB_CUDA(cudaFuncSetAttribute(latent_out_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSmemMax - 8192));
    attr_set = true;
  }
  const dim3 gq((unsigned)((a.m.kv_rank + LQ_N - 1) / LQ_N), (unsigned)a.m.heads, (unsigned)a.chunks.count);
  RB_CUDA(launch_k(latent_q_kernel, gq, dim3(256), q_smem, c->stream, c->use_pdl, a));
  const dim3 ga((unsigned)a.kv_splits, (unsigned)(a.tiles.count * cf.subtiles), (unsigned)((a.m.heads + cf.heads_per - 1) / cf.heads_per));
  if (mt == 1) RB_CUDA(launch_k(latent_attn_kernel<1>, ga, dim3(288), smem, c->stream, c->use_pdl, *a.tm_cache, a, cf));
  else RB_CUDA(launch_k(latent_attn_kernel<2>, ga, dim3(288), smem, c->stream, c->use_pdl, *a.tm_cache, a, cf));
  const dim3 go((unsigned)((a.m.vdim + LO_N - 1) / LO_N), (unsigned)a.m.heads, (unsigned)(a.chunks.list ? (int64_t)a.chunks.count * LO_PARTS : (a.rows + LO_ROWS - 1) / LO_ROWS));
  RB_CUDA(launch_k(latent_out_kernel, go, dim3(256), o_smem, c->stream, c->use_pdl, a));
  g_launch_total += 3;
  return REWB200_OK;
}

int gather_rows_launch(Ctx* c, const void* src, const int* index, void* dst, int64_t n, int64_t width, int dtype) {
  if (n == 0) return REWB200_OK;
  if (dtype == REWB200_BF16)
    RB_CUDA(launch_k(gather_rows_kernel<bf16>, dim3((unsigned)n), dim3(128), 0, c->stream, c->use_pdl, (const bf16*)src, index, (bf16*)dst, width));
  else
    RB_CUDA(launch_k(gather_rows_kernel<float>, dim3((unsigned)n), dim3(128), 0, c->stream, c->use_pdl, (const float*)src, index, (float*)dst, width));
  ++g_launch_total;
  return REWB200_OK;
}

}  // namespace rewb
