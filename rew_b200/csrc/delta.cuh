// Gated delta rule of layered models: a state S [dim, vdim] per head and sequence; a token decays it by one number g, corrects
// it towards its value at its key and reads it with its query:
//   S <- g S,   u = beta (v - S^T k),   S <- S + k u^T,   o = S^T q
// with unit keys and queries shared by groups of heads.  Argument structs and launchers of delta.cu (token by token: decoded
// tokens, small portions, f32 models) and delta_chunk.cu (large prompt portions on the tensor cores).
#pragma once
#include "gla.cuh"

namespace rewb {

struct DeltaDims {
  int heads, kv_heads, dim, vdim;
  const float* rate;       // [heads] exp(A_log)
  const float* dt_bias;    // [heads]
  const float* norm;       // [vdim]
  float scale;             // of the output
};
inline __host__ __device__ int64_t delta_channels(const DeltaDims& m) { return 2 * (int64_t)m.kv_heads * m.dim + (int64_t)m.heads * m.vdim; }

struct DeltaArgs {
  DeltaDims m;
  const GlaPortion* list;  // nullptr: one token for each of `count` lanes from b0 on, at position pos0[lane]
  int count;
  const int* pos0;
  int b0;
  const int2* chunks;      // large portions: (first row, tokens) of every chunk
  int n_chunks;
  uint8_t* work;           // ... scratch, delta_chunk_bytes a chunk
  const void* x;           // [rows][ldx] act dtype: q kv_heads*dim | k kv_heads*dim | v heads*vdim as they leave the convolution
  int64_t ldx;
  // gate heads*vdim | beta heads | decay heads: columns of the projection's slabs [nsplit][rows][ld]
  const float* partial;
  int nsplit;
  int64_t split_stride, ld;
  float eps;
  float* state;            // [lanes][heads][dim][ldv] f32
  int ldv;
  void* out;               // [rows][ldo] act dtype, head-major columns: normed, gated, scaled
  int64_t ldo;
  int dtype;
  int early;               // captured decode step: state and positions predate the step
  int* status;
};
int delta_recurrent_launch(Ctx* c, const DeltaArgs& a);
int delta_rate_launch(Ctx* c, float* a_log, int64_t n);   // exp in place
bool delta_chunk_ok(const DeltaDims& m);
int delta_chunks(int n);                                  // chunks of a portion of n tokens
int2 delta_chunk_rows(const GlaPortion& p, int i);        // first row and tokens of its i-th chunk
size_t delta_chunk_bytes(const DeltaDims& m);             // scratch of one chunk, all heads
int delta_chunk_launch(Ctx* c, const DeltaArgs& a);

}  // namespace rewb
