// Grouped-query attention of large prompt portions: the tcgen05 kernel of flash_tc.cuh on the cache's pages, with a sink and,
// where the layer has one, a bias by distance.  With a bias, key tiles further back than the bias table reaches add one number; the others read the table in
// shared memory, whose entries for keys after the query are -inf.
#include <algorithm>

#include "flash_tc.cuh"
#include "gqa.cuh"

namespace rewb {

namespace {

template <bool BIAS>
struct GqaPolicy {
  static constexpr bool kBias = BIAS;
  GqaPrefillArgs a;
  int nb;                  // distances the bias tells apart
  int heads, vdim;
  float scale;
  const float* gate;
  bf16* out;
  int64_t ldo;
  int* status;

  __device__ __forceinline__ GqaTile tile(int i, int skip) const {
    GqaTile t = a.tiles[i];
    t.row0 += skip;
    t.n -= skip;
    t.pos0 += skip;
    return t;
  }
  __device__ __forceinline__ int window() const { return 0; }
  __device__ __forceinline__ int k_base(const GqaTile&) const { return 0; }
  __device__ __forceinline__ int n_bias() const { return nb; }
  __device__ __forceinline__ float sink(int head) const { return a.m.sink ? a.m.sink[head] : -INFINITY; }
  __device__ __forceinline__ void bias_table(int head, float* tab, int tid, int nt) const {
    for (int i = tid; i < flash::bias_slots(nb); i += nt) {
      const int d = i - flash::BIAS_PAD;
      tab[i] = d < 0 ? -INFINITY : a.m.bias[(int64_t)head * nb + min(d, nb - 1)] * flash::LOG2E;
    }
  }
  __device__ __forceinline__ uint4 q_chunk(const GqaTile& t, int qi, int head, int box, int c) const {
    const int f = box * 64 + c;
    if (f >= a.m.dim) return make_uint4(0, 0, 0, 0);
    return *reinterpret_cast<const uint4*>(a.q + (int64_t)(t.row0 + qi) * a.ldq + (int64_t)head * a.m.dim + f);
  }
  // a tile of 128 keys is two pages
  __device__ __forceinline__ void pages(uint8_t* dst, const CUtensorMap& tm, uint64_t* bar, const GqaTile& t, int head, int j, int boxes) const {
    const int hk = head / (a.m.heads / a.m.kv_heads);
#pragma unroll
    for (int p = 0; p < 2; ++p) {
      const int page = a.block_table[(int64_t)t.lane * a.max_pages + min(2 * j + p, a.max_pages - 1)];
      for (int b = 0; b < boxes; ++b) tma_load_2d(dst + b * flash::BOX_BYTES + p * 8192, &tm, bar, b * 64, (page * a.m.kv_heads + hk) * 64);
    }
  }
  __device__ __forceinline__ void load_k(uint8_t* dst, const CUtensorMap& tm_k, const CUtensorMap&, uint64_t* bar, const GqaTile& t, int head, int j, int,
                                         const flash::Cfg& cf) const {
    pages(dst, tm_k, bar, t, head, j, cf.nb_k);
  }
  __device__ __forceinline__ void load_v(uint8_t* dst, const CUtensorMap&, const CUtensorMap& tm_v, uint64_t* bar, const GqaTile& t, int head, int j, int,
                                         const flash::Cfg& cf) const {
    pages(dst, tm_v, bar, t, head, j, cf.nb_v);
  }
};

size_t table_bytes(const GqaDims& m) { return m.bias ? (size_t)flash::bias_slots(m.n_bias) * sizeof(float) : 0; }

}  // namespace

bool gqa_prefill_ok(const GqaDims& m) {
  return m.dim % 8 == 0 && m.vdim % 8 == 0 && m.dim <= 256 && m.vdim <= 128 && m.scale > 0.f && table_bytes(m) <= 24 * 1024;
}

int gqa_prefill_launch(Ctx* c, const GqaPrefillArgs& a) {
  if (a.count == 0) return REWB200_OK;
  RB_REQUIRE(gqa_prefill_ok(a.m), "grouped-query attention: head sizes without a tcgen05 kernel");
  auto go = [&](auto p, size_t table) {
    return flash::launch(c, p, *a.tm_k, *a.tm_v, a.count, (a.m.dim + 63) / 64, (a.m.vdim + 63) / 64, table);
  };
  const float* gate = a.m.gate ? a.gate : nullptr;
  if (a.m.bias) return go(GqaPolicy<true>{a, a.m.n_bias, a.m.heads, a.m.vdim, a.m.scale, gate, a.out, a.ldo, a.status}, table_bytes(a.m));
  return go(GqaPolicy<false>{a, 1, a.m.heads, a.m.vdim, a.m.scale, gate, a.out, a.ldo, a.status}, 0);
}

}  // namespace rewb
