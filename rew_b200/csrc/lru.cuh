// Linear recurrent unit of layered models: S <- a S + sqrt(1 - a^2) i u per channel, a = exp(decay r), with gates r and i and
// an output S gelu(y).  Argument structs and launcher of lru.cu.
#pragma once
#include "gla.cuh"

namespace rewb {

struct LruDims {
  int blocks, n, ldn;      // channels of a block, padded to a multiple of 8
  const float* decay;      // [width] -8 softplus(lam)
  const float* y_bias;     // [width]
  float scale;             // of the output
};
struct LruArgs {
  LruDims m;
  const GlaPortion* list;  // nullptr: one token for each of `count` lanes from b0 on, at position pos0[lane]
  int count;
  int longest;             // tokens of the longest portion
  const int* pos0;
  int b0;
  int64_t rows;
  const float* gates;      // [blocks][rows][2 ldn] r | i ahead of their sigmoids
  const void* u;           // [blocks][rows][ldn] act dtype
  const float* partial;    // y, first of `width` columns of the projection's slabs [nsplit][rows][ld]
  int nsplit;
  int64_t split_stride, ld;
  float* state;            // [lanes][width] f32
  void* out;               // [rows][ldo] act dtype
  int64_t ldo;
  int dtype;
  int early;               // captured decode step: state and positions predate the step
};
int lru_launch(Ctx* c, const LruArgs& a);
int lru_decay_launch(Ctx* c, float* lam, int64_t n);   // -8 softplus(lam) in place

}  // namespace rewb
