// Latent attention kernels (see latent.cuh): the fused post-processing of the input projection, and attention on the
// cached latents.  Scores, softmax, norms, rotations and gates are f32 throughout.
#include <math.h>

#include "latent.cuh"
#include "ptx.cuh"

namespace rewb {

extern int64_t g_launch_total;

namespace {

constexpr int PAGE_TOKENS = 64;

template <typename T> __device__ __forceinline__ float ldf(T v);
template <> __device__ __forceinline__ float ldf<float>(float v) { return v; }
template <> __device__ __forceinline__ float ldf<bf16>(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T stf(float v);
template <> __device__ __forceinline__ float stf<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 stf<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ int row_lane(const RowMap& m, int64_t row) {
  return m.row_lane ? m.row_lane[row] : m.b0 + (int)(row / m.S);
}
__device__ __forceinline__ int row_pos(const RowMap& m, int64_t row) {
  return m.row_pos ? m.row_pos[row] : m.pos0[m.b0 + row / m.S] + (int)(row % m.S);
}
__device__ __forceinline__ int2 tile_rows(const RowTiles& t, int i) {
  if (t.list) return t.list[i];
  const int per_lane = (t.S + t.per_tile - 1) / t.per_tile;
  const int lane = i / per_lane, k = (i % per_lane) * t.per_tile;
  return make_int2(lane * t.S + k, min(t.per_tile, t.S - k));
}
__device__ __forceinline__ float2 rotate(float2 v, float2 cs) {
  return make_float2(v.x * cs.x - v.y * cs.y, v.y * cs.x + v.x * cs.y);
}

__device__ __forceinline__ float block_sum256(float v, float* red) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
  const int w = threadIdx.x >> 5;
  __syncthreads();
  if ((threadIdx.x & 31) == 0) red[w] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < 8; ++i) t += red[i];
  return t;
}

// One CTA per row.
template <typename T>
__global__ void __launch_bounds__(256) latent_post_kernel(LatentPostArgs a) {
  extern __shared__ float sx[];
  __shared__ float red[8];
  pdl_launch_dependents();
  pdl_wait();
  const int64_t row = blockIdx.x;
  const int nq = a.m.q_rank, nc = a.m.kv_rank, nr = a.m.rot_dim, n = nq + nc + nr + (a.m.gate ? a.m.heads : 0);
  const float* p = a.partial + row * a.ld;
  float sq = 0.f, sc = 0.f;
  for (int i = threadIdx.x; i < n; i += 256) {
    float v = 0.f;
    for (int s = 0; s < a.nsplit; ++s) v += p[s * a.split_stride + i];
    sx[i] = v;
    if (i < nq) sq += v * v;
    else if (i < nq + nc) sc += v * v;
  }
  sq = block_sum256(sq, red);
  sc = block_sum256(sc, red);
  const float rq = sqrtf(sq / (float)nq + a.eps), rc = sqrtf(sc / (float)nc + a.eps);
  const int lane = row_lane(a.map, row), pos = row_pos(a.map, row);
  const bool ok = pos >= 0 && pos < a.capacity && pos < a.m.max_pos;
  if (!ok && threadIdx.x == 0) atomicExch(a.status, KS_BAD_INDEX);
  T* cq = reinterpret_cast<T*>(a.cq) + row * a.ldcq;
  for (int i = threadIdx.x; i < nq; i += 256) cq[i] = stf<T>(a.q_norm[i] * (sx[i] / rq));
  if (a.m.gate)
    for (int i = threadIdx.x; i < a.m.heads; i += 256) a.gate[row * a.m.heads + i] = 1.0f / (1.0f + expf(-sx[nq + nc + nr + i]));
  if (!ok) return;
  const int page = a.block_table[(int64_t)lane * a.max_pages + pos / PAGE_TOKENS];
  T* cr = reinterpret_cast<T*>(a.cache) + ((int64_t)page * PAGE_TOKENS + pos % PAGE_TOKENS) * a.ldc;
  for (int i = threadIdx.x; i < nc; i += 256) cr[i] = stf<T>(a.kv_norm[i] * (sx[nq + i] / rc));
  const int half = a.m.rope_dims / 2;
  for (int i = threadIdx.x; i < half; i += 256) {
    const float2 v = rotate(make_float2(sx[nq + nc + 2 * i], sx[nq + nc + 2 * i + 1]), a.m.rope[(int64_t)pos * half + i]);
    cr[nc + 2 * i] = stf<T>(v.x);
    cr[nc + 2 * i + 1] = stf<T>(v.y);
  }
  for (int i = 2 * half + threadIdx.x; i < nr; i += 256) cr[nc + i] = stf<T>(sx[nq + nc + i]);
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
  float mx = -INFINITY, l = 0.f;
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
  const size_t smem = (size_t)(a.m.q_rank + a.m.kv_rank + a.m.rot_dim + a.m.heads) * sizeof(float);
  RB_REQUIRE(smem <= 48 * 1024, "latent attention: the input projection is wider than 12288 columns");
  if (a.dtype == REWB200_BF16)
    RB_CUDA(launch_k(latent_post_kernel<bf16>, dim3((unsigned)rows), dim3(256), smem, c->stream, c->use_pdl, a));
  else
    RB_CUDA(launch_k(latent_post_kernel<float>, dim3((unsigned)rows), dim3(256), smem, c->stream, c->use_pdl, a));
  ++g_launch_total;
  return REWB200_OK;
}

int latent_kv_splits(Ctx* c, const LatentDims& m, int64_t tiles, int64_t max_ctx) {
  (void)c; (void)m; (void)tiles; (void)max_ctx;
  return 1;
}

int latent_attn_absorbed_launch(Ctx* c, const LatentAttnArgs& a) {
  if (a.tiles.count == 0) return REWB200_OK;
  return a.dtype == REWB200_BF16 ? plain_launch<bf16>(c, a) : plain_launch<float>(c, a);
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
