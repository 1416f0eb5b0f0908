// Grouped-query attention of layered models: a short causal convolution over time on queries and keys, per-head RMS norms,
// a query temperature that grows with the position, rotated features, a learned bias per head and distance bucket, a number
// per head in the softmax denominator ("sink"), an output gate per head, each of them optional.  Layers with a window, kept first
// keys, mixed heads or a gate per feature run the kernels of gqa_mix.cuh.  Argument structs and launchers of gqa.cu and
// gqa_prefill.cu.
//
// Caches: keys [pages][kv_heads][64][ldk], values [pages][kv_heads][64][ldv].
#pragma once
#include "steprows.cuh"

namespace rewb {

struct GqaDims {
  int heads, kv_heads, dim, vdim;
  int own_kv;              // 0: another layer's keys and values
  int gate;
  float scale;
  const float* q_norm;     // [dim] or nullptr: no norm
  const float* k_norm;
  int temp_every;          // queries times 1 + temp_coef ln(floor((p + 1) / temp_every) + 1); 0: no temperature
  float temp_coef;
  const float* bias;       // [heads][n_bias] by distance; the last entry holds for every longer distance; nullptr: none
  int n_bias;
  const float* sink;       // [heads] or nullptr
  int v_from_k;            // the values are the keys as they leave the convolution: no value projection
  int taps;                // of the convolution per channel of queries and keys; 0: none
  const float* conv;       // [taps][gqa_channels]: the weight of the value taps - 1 - j tokens ago is row j
  int rope_dims;           // rotated features at the start of a head, pairs (i, i + rope_dims / 2); 0: none
  const float2* rope;      // [max_pos][rope_dims / 2] (cos, sin)
  int pairs;               // rotated features are pairs (2i, 2i + 1)
  int v_norm;              // values are divided by their root mean square
  const float* in_bias;    // by column of the projection's queries, keys and values, or nullptr (no convolution then)
  int window, keep_first;  // keys a query sees, itself included (0: all), and the first keys of the sequence it sees besides
  const float* talk;       // [heads][heads] mixes the heads' weights after the softmax, or nullptr
  int talk_wide;           // it has numbers that f16 has not
  int gate_elem;           // the output gate is per feature
  float out_scale;         // of the output
};
// What the kernels of gqa_mix.cuh are for.
inline bool gqa_is_mixed(const GqaDims& m) { return m.window > 0 || m.talk || m.gate_elem || m.out_scale != 1.0f; }

// Channels of the projection the convolution runs on: queries, then keys of its own.
inline __host__ __device__ int64_t gqa_channels(const GqaDims& m) { return (int64_t)(m.heads + (m.own_kv ? m.kv_heads : 0)) * m.dim; }
// f32 elements of convolution state per sequence: the projected values of the last taps - 1 tokens, that of position p in
// slot p % (taps - 1).  A portion that starts at position 0 reads none of them, so a lane needs no clearing.
inline int64_t gqa_state_elems(const GqaDims& m) { return m.taps > 1 ? (m.taps - 1) * gqa_channels(m) : 0; }

// Finishes the fused input projection [q | k | v | gate] (q | gate without keys of its own, no v where the values are the
// keys): sums the split-K slabs, adds biases, runs the convolution, norms queries, keys and values, applies the temperature,
// rotates, appends keys and values to the cache.  A gate per feature is left to the kernel that reads it.
struct GqaPostArgs {
  GqaDims m;
  const float* partial;    // [nsplit][rows][ld]
  int nsplit;
  int64_t split_stride, ld;
  float eps;
  RowMap map;
  void* q;                 // [rows][ldq] act dtype
  int64_t ldq;
  float* gate;             // [rows][heads]
  void *kc, *vc;
  int64_t ldk, ldv;
  const int* block_table;
  int max_pages, capacity;
  int dtype;
  int early;               // captured decode step: positions predate the step
  float* state;            // convolution state [lanes][taps - 1][gqa_channels], or nullptr
  // Rows whose values enter the state: every row of a step of single tokens (tails == nullptr), written on the way, or the
  // last rows of every portion, (row, rows of the portion behind it), written by gqa_conv_state_launch.
  const int2* tails;
  int n_tails;
  int* status;
};
int gqa_post_launch(Ctx* c, const GqaPostArgs& a, int64_t rows);
int gqa_conv_state_launch(Ctx* c, const GqaPostArgs& a);

// Attention of the rows in `tiles` (decoded tokens, small portions).
struct GqaAttnArgs {
  GqaDims m;
  RowMap map;
  RowTiles tiles;
  int max_tile_rows;
  const void* q;
  int64_t ldq;
  const float* gate;
  void* out;               // [rows][ldo] act dtype, head-major columns
  int64_t ldo;
  const void *kc, *vc;
  const CUtensorMap *tm_k, *tm_v;  // bf16: box 64 x 64
  int64_t ldk, ldv;
  const int* block_table;
  int max_pages;
  int dtype;
  float* o_part;           // scratch [rows][heads][kv splits][vdim], not yet divided by the row sum
  float2* ml;              // scratch [rows][heads][kv splits] running maximum (base 2) and sum
  int kv_splits;
  int early_kv;            // captured decode step: cache pages other than the newest may be loaded ahead of the stream dependency
  int* status;
};
int gqa_attn_launch(Ctx* c, const GqaAttnArgs& a);
int gqa_kv_splits(Ctx* c, const GqaDims& m, int64_t tiles, int64_t max_ctx);

// Attention of large prompt portions on tcgen05; one tile = up to 256 queries of one portion.
struct GqaTile {
  int row0, n, pos0, lane;
};
struct GqaPrefillArgs {
  GqaDims m;
  const GqaTile* tiles;
  int count;
  const bf16* q;
  int64_t ldq;
  const float* gate;
  bf16* out;
  int64_t ldo;
  const CUtensorMap *tm_k, *tm_v;
  const int* block_table;
  int max_pages;
  int* status;
};
bool gqa_prefill_ok(const GqaDims& m);
int gqa_prefill_launch(Ctx* c, const GqaPrefillArgs& a);

}  // namespace rewb
