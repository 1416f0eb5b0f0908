// Grouped-query attention whose heads meet after the softmax: head h weighs keys with sum_g T[h, g] (softmax of head g), over a
// sliding window and the first keys of the sequence, with a gate per feature on the output; each of them optional.  The
// weights of all heads must be known, normalised, before any head can read its values, so scores and values are separate
// launches with the scores between them.  Argument structs and launchers of gqa_mix.cu and gqa_mix_prefill.cu.
#pragma once
#include "gqa.cuh"

namespace rewb {

struct GqaMixArgs {
  GqaDims m;
  RowMap map;
  RowTiles tiles;          // runs of rows (decoded tokens, small portions)
  int max_tile_rows;
  int64_t rows;            // of the step
  const void* q;
  int64_t ldq;
  const float* gate;       // gate columns of the projection's slabs [nsplit][rows][ld] (gate_elem), or nullptr
  int nsplit;
  int64_t split_stride, ld;
  const float* gate_head;  // [rows][heads] (a gate per head), or nullptr
  void* out;               // [rows][ldo] act dtype, head-major columns
  int64_t ldo;
  const void *kc, *vc;
  const CUtensorMap *tm_k, *tm_v;
  int64_t ldk, ldv;
  const int* block_table;
  int max_pages;
  int dtype;
  float* work;             // scratch of work_bytes
  size_t work_bytes;
  int early_kv;            // captured decode step: cache pages other than the newest may be loaded ahead of the stream dependency
  int* status;
};
// Scratch that a step of `rows` rows in `tiles` tiles wants at most, contexts up to max_ctx.
size_t gqa_mix_bytes(Ctx* c, const GqaDims& m, int dtype, int64_t rows, int64_t tiles, int64_t max_tile_rows, int64_t max_ctx);
int gqa_mix_launch(Ctx* c, const GqaMixArgs& a);

// Large prompt portions on tcgen05; tiles as in GqaPrefillArgs, talk_host: the mixing matrix on the host (nullptr: none), lse:
// scratch [rows][heads].  Of `a`, the tiles and the scratch are not read.
bool gqa_mix_prefill_ok(const GqaDims& m);
int gqa_mix_prefill_launch(Ctx* c, const GqaMixArgs& a, const GqaTile* tiles, int count, const float* talk_host, float* lse);

}  // namespace rewb
