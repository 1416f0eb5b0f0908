// Gated linear attention of layered models: a state S [dim, vdim] per head and sequence, S <- diag(alpha_t) S + k_t v_t^T,
// o_t = S^T q_t, with a decay alpha per key channel.  Argument structs and launchers of gla.cu (token by token: decoded
// tokens, small portions, f32 models) and gla_chunk.cu (large prompt portions on the tensor cores).
#pragma once
#include "steprows.cuh"

namespace rewb {

struct GlaDims {
  int heads, dim, vdim, rank;
  float tau;
  const float* a2;         // [rank][heads * dim] second decay projection
  const float* a2_b;       // [heads * dim]
  const float* norm;       // [vdim]
};

// A portion of a step: rows row0 .. row0 + n - 1 are the tokens at positions pos0 .. of `lane`.
struct GlaPortion {
  int row0, n, pos0, lane;
  int chunk0;              // large portions: the first of its chunks in GlaArgs::chunks
};

struct GlaArgs {
  GlaDims m;
  const GlaPortion* list;  // nullptr: one token for each of `count` lanes from b0 on, at position pos0[lane]
  int count;
  const int* pos0;
  int b0;
  const int2* chunks;      // large portions: (first row, tokens) of every chunk
  int n_chunks;
  uint8_t* work;           // ... scratch, gla_chunk_bytes a chunk
  // fused input projection [q heads*dim | k heads*dim | v heads*vdim | gate heads*vdim | decay rank], split-K slabs
  const float* partial;    // [nsplit][rows][ld]
  int nsplit;
  int64_t split_stride, ld;
  float eps;
  float* state;            // [lanes][heads][dim][ldv] f32
  int ldv;
  void* out;               // [rows][ldo] act dtype, head-major columns: normed, gated
  int64_t ldo;
  int dtype;
  int early;               // captured decode step: state and positions predate the step
  int* status;
};
int64_t gla_state_ld(int vdim);
int gla_recurrent_launch(Ctx* c, const GlaArgs& a);
bool gla_chunk_ok(const GlaDims& m);
int gla_chunks(int n);                                  // chunks of a portion of n tokens
int2 gla_chunk_rows(const GlaPortion& p, int i);        // first row and tokens of its i-th chunk
size_t gla_chunk_bytes(const GlaDims& m);               // scratch of one chunk, all heads
int gla_chunk_launch(Ctx* c, const GlaArgs& a);

}  // namespace rewb
