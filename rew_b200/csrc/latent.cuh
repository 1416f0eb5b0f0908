// Latent attention (multi-head attention whose keys and values are linear in a cached low-rank latent): argument
// structs and launchers of latent.cu.
//
// Per token the cache row holds [c (kv_rank) | k_rot (rot_dim)], shared by all heads.  A head's score against a key
// is q_nope . (W_uk c) + q_rot . k_rot = [W_uk^T q_nope | q_rot] . [c | k_rot], and its output is
// W_uv (sum_j p_j c_j), so attention can run on the cache rows themselves ("absorbed": small steps, decode) or on
// keys and values expanded from them per head (large prompt portions).
#pragma once
#include "steprows.cuh"

namespace rewb {

constexpr int kChunkRows = 64;   // RowTiles of LatentAttnArgs::chunks

struct LatentDims {
  int heads, dim, rot_dim, vdim, q_rank, kv_rank;
  int rope_dims;           // rotated features of the rot_dim part (interleaved pairs), the rest passes unchanged
  int window;              // keys a query sees, itself included; 0: all
  int gate;                // per-head output gate
  float scale;
  const float2* rope;      // [max_pos][rope_dims / 2] (cos, sin)
  int max_pos;
  int own_kv;              // 0: another layer's cached latents
  const float* sink;       // [heads] a score without a key or value in the softmax denominator, or nullptr
};

// Finishes the fused input projection [q_rank | kv_rank | rot_dim | heads] (q_rank | heads without latents of its own): sums the split-K slabs, norms the query
// latent and the key/value latent, rotates the shared key part, appends [c | k_rot] to the cache, applies the
// sigmoid of the output gate.
struct LatentPostArgs {
  LatentDims m;
  const float* partial;    // [nsplit][rows][ld]
  int nsplit;
  int64_t split_stride, ld;
  const float *q_norm, *kv_norm;
  float eps;
  RowMap map;
  void* cq;                // [rows][ldcq] act dtype
  int64_t ldcq;
  float* gate;             // [rows][heads]
  void* cache;             // [pages][64][ldc]
  const int* block_table;  // [lanes][max_pages]
  int max_pages, capacity;
  int64_t ldc;
  int dtype;
  int early;               // captured decode step: positions predate the step
  int* status;
};
int latent_post_launch(Ctx* c, const LatentPostArgs& a, int64_t rows);

// Absorbed attention of the rows in `tiles`.
struct LatentAttnArgs {
  LatentDims m;
  RowMap map;
  RowTiles tiles;          // runs of rows of one lane
  int max_tile_rows;       // rows of the longest tile
  RowTiles chunks;         // the same rows in runs of up to kChunkRows, whatever their lanes
  int64_t rows;            // rows of the whole step
  // queries: either split-K slabs f32 [nsplit][rows][ldq] or (nsplit == 0) act dtype [rows][ldq]
  const void* q;
  int nsplit;
  int64_t split_stride, ldq;
  const void* ukv;         // [kv_rank][ld_ukv] act dtype: columns heads*dim of keys, then heads*vdim of values
  int64_t ld_ukv;
  void* qeff;              // scratch [rows][heads][ldc] act dtype
  float* olat;             // scratch [rows][heads][kv splits][kv_rank] f32, not yet divided by the row sum
  float2* ml;              // scratch [rows][heads][kv splits] running maximum and sum
  int kv_splits;
  const float* gate;       // [rows][heads]
  void* out;               // [rows][ldo] act dtype, head-major columns
  int64_t ldo;
  const void* cache;
  const CUtensorMap* tm_cache;  // bf16: [pages * 64][ldc], box 64 x 64
  const int* block_table;
  int max_pages;
  int64_t ldc;
  int dtype;
  int early_kv;            // captured decode step: cache pages other than the newest may be loaded ahead of the stream dependency
  int* status;
};
int latent_attn_absorbed_launch(Ctx* c, const LatentAttnArgs& a);
int latent_kv_splits(Ctx* c, const LatentDims& m, int64_t tiles, int64_t max_ctx);

// Expanded attention of large prompt portions: keys and values of every head are computed from the gathered cache rows by
// one Linear, then attention runs on them with tcgen05.  One tile = up to 256 queries of one portion.
struct ExpTile {
  int row0, n;     // rows of the step
  int pos0;        // position of the first one
  int key0;        // first position of the portion's gathered keys
  int off;         // row of the gathered buffers = position + off
  int pad[3];
};
struct LatentExpArgs {
  LatentDims m;
  const ExpTile* tiles;
  int count;
  const bf16* q;           // [rows][ldq], unrotated
  int64_t ldq;
  const float* gate;       // [rows][heads]
  bf16* out;               // [rows][ldo]
  int64_t ldo;
  const bf16* kv;          // [keys][ldkv]: heads*dim of keys, then heads*vdim of values
  int64_t ldkv;
  const bf16* lat;         // [keys][ldc] gathered cache rows (their rotated part is the shared key part)
  int64_t ldc, keys;
  int* status;
};
bool latent_expanded_ok(const LatentDims& m);
int latent_attn_expanded_launch(Ctx* c, const LatentExpArgs& a);
// dst[i] = cache row of position index[i].y of lane index[i].x
int latent_gather_launch(Ctx* c, const bf16* cache, const int* block_table, int max_pages, int64_t ldc, const int2* index, bf16* dst, int64_t n);

// Gathers rows of the step: dst[i] = src[index[i]] (width elements of `dtype`).
int gather_rows_launch(Ctx* c, const void* src, const int* index, void* dst, int64_t n, int64_t width, int dtype);

}  // namespace rewb
