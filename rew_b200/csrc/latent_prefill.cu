// Latent attention of large prompt portions on keys and values expanded per head: the tcgen05 kernel of flash_tc.cuh.  The
// rotated features all heads share come from the gathered cache rows; queries are rotated on the way in.
#include "flash_tc.cuh"
#include "latent.cuh"

namespace rewb {

namespace {

struct LatentPolicy {
  static constexpr bool kBias = false;
  LatentExpArgs a;
  int nb_n;                // boxes of unrotated features
  int heads, vdim;
  float scale;
  const float* gate;
  bf16* out;
  int64_t ldo;
  int* status;

  __device__ __forceinline__ ExpTile tile(int i, int skip) const {
    ExpTile t = a.tiles[i];
    t.row0 += skip;
    t.n -= skip;
    t.pos0 += skip;
    return t;
  }
  __device__ __forceinline__ int window() const { return a.m.window; }
  __device__ __forceinline__ int k_base(const ExpTile& t) const { return max(t.key0, a.m.window > 0 ? t.pos0 - a.m.window + 1 : 0); }
  __device__ __forceinline__ int n_bias() const { return 1; }
  __device__ __forceinline__ float sink(int head) const { return a.m.sink ? a.m.sink[head] : -INFINITY; }
  __device__ __forceinline__ uint4 q_chunk(const ExpTile& t, int qi, int head, int box, int c) const {
    const bf16* qp = a.q + (int64_t)(t.row0 + qi) * a.ldq + (int64_t)head * (a.m.dim + a.m.rot_dim);
    uint4 v = make_uint4(0, 0, 0, 0);
    if (box < nb_n) {
      const int f = box * 64 + c;
      if (f < a.m.dim) v = *reinterpret_cast<const uint4*>(qp + f);
      return v;
    }
    const int f = (box - nb_n) * 64 + c, half_r = a.m.rope_dims / 2;
    if (f >= a.m.rot_dim) return v;
    const float2* rope = a.m.rope + (int64_t)min(t.pos0 + qi, a.m.max_pos - 1) * half_r;
    v = *reinterpret_cast<const uint4*>(qp + a.m.dim + f);
    uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int p = f / 2 + e;
      if (p < half_r) {
        const __nv_bfloat162 x = *reinterpret_cast<const __nv_bfloat162*>(&w[e]);
        const float2 cs = rope[p];
        const float u = __low2float(x), s = __high2float(x);
        w[e] = pack_bf16(u * cs.x - s * cs.y, s * cs.x + u * cs.y);
      }
    }
    return make_uint4(w[0], w[1], w[2], w[3]);
  }
  __device__ __forceinline__ void load_k(uint8_t* dst, const CUtensorMap& tm_kv, const CUtensorMap& tm_lat, uint64_t* bar, const ExpTile& t, int head,
                                         int j, int k_base, const flash::Cfg& cf) const {
    const int krow = k_base + j * 128 + t.off;
    for (int b = 0; b < nb_n; ++b) tma_load_2d(dst + b * flash::BOX_BYTES, &tm_kv, bar, head * a.m.dim + b * 64, krow);
    for (int b = nb_n; b < cf.nb_k; ++b) tma_load_2d(dst + b * flash::BOX_BYTES, &tm_lat, bar, a.m.kv_rank + (b - nb_n) * 64, krow);
  }
  __device__ __forceinline__ void load_v(uint8_t* dst, const CUtensorMap& tm_kv, const CUtensorMap&, uint64_t* bar, const ExpTile& t, int head, int j,
                                         int k_base, const flash::Cfg& cf) const {
    const int krow = k_base + j * 128 + t.off;
    for (int b = 0; b < cf.nb_v; ++b) tma_load_2d(dst + b * flash::BOX_BYTES, &tm_kv, bar, heads * a.m.dim + head * vdim + b * 64, krow);
  }
};

__global__ void __launch_bounds__(256) latent_gather_kernel(const bf16* cache, const int* block_table, int max_pages, int64_t ldc, const int2* index,
                                                            bf16* dst, int64_t n) {
  pdl_launch_dependents();
  pdl_wait();
  const int64_t i = (int64_t)blockIdx.x * 8 + (threadIdx.x >> 5);
  if (i >= n) return;
  const int2 lp = index[i];
  const int page = block_table[(int64_t)lp.x * max_pages + lp.y / 64];
  const uint4* src = reinterpret_cast<const uint4*>(cache + ((int64_t)page * 64 + lp.y % 64) * ldc);
  uint4* d = reinterpret_cast<uint4*>(dst + i * ldc);
  for (int c = threadIdx.x & 31; c < ldc / 8; c += 32) d[c] = src[c];
}

}  // namespace

// Head sizes the kernel takes: whole 16-byte chunks everywhere a TMA load starts, score features in at most four boxes,
// values in at most two.
bool latent_expanded_ok(const LatentDims& m) {
  const int nb = (m.dim + 63) / 64 + (m.rot_dim + 63) / 64;
  return m.dim % 8 == 0 && m.rot_dim % 8 == 0 && m.vdim % 8 == 0 && m.kv_rank % 8 == 0 && m.rope_dims % 2 == 0 && nb <= 4 &&
         m.vdim <= 128 && m.scale > 0.f;
}

int latent_attn_expanded_launch(Ctx* c, const LatentExpArgs& a) {
  if (a.count == 0) return REWB200_OK;
  RB_REQUIRE(latent_expanded_ok(a.m), "latent attention: head sizes without an expanded kernel");
  CUtensorMap tm_kv, tm_lat;
  RB_TRY(make_tmap_2d_bf16(&tm_kv, a.kv, (uint64_t)a.m.heads * (a.m.dim + a.m.vdim), (uint64_t)a.keys, (uint64_t)a.ldkv * 2, 64, 128));
  RB_TRY(make_tmap_2d_bf16(&tm_lat, a.lat, (uint64_t)a.m.kv_rank + a.m.rot_dim, (uint64_t)a.keys, (uint64_t)a.ldc * 2, 64, 128));
  const int nb_n = (a.m.dim + 63) / 64;
  const LatentPolicy p = {a, nb_n, a.m.heads, a.m.vdim, a.m.scale, a.m.gate ? a.gate : nullptr, a.out, a.ldo, a.status};
  return flash::launch(c, p, tm_kv, tm_lat, a.count, nb_n + (a.m.rot_dim + 63) / 64, (a.m.vdim + 63) / 64, 0);
}

int latent_gather_launch(Ctx* c, const bf16* cache, const int* block_table, int max_pages, int64_t ldc, const int2* index, bf16* dst, int64_t n) {
  if (n == 0) return REWB200_OK;
  RB_CUDA(launch_k(latent_gather_kernel, dim3((unsigned)((n + 7) / 8)), dim3(256), 0, c->stream, c->use_pdl, cache, block_table, max_pages, ldc, index, dst, n));
  ++g_launch_total;
  return REWB200_OK;
}

}  // namespace rewb
