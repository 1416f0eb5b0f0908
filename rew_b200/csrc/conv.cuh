// Short causal convolution over time, per channel, of a range of columns of a projection.  Argument structs and launchers of
// conv.cu.
#pragma once
#include "steprows.cuh"

namespace rewb {

struct ConvDims {
  int64_t channels;
  int taps;
  const float* w;          // [taps][channels]: the weight of the value taps - 1 - j tokens ago is row j
  const float* in_bias;    // [channels] added to the projection ahead of the convolution, or nullptr
  const float* bias;       // [channels] added behind it, or nullptr
  int silu;
};
// f32 elements of state per sequence: the inputs of the last taps - 1 tokens, that of position p in slot p % (taps - 1).  A
// portion that starts at position 0 reads none of them, so a lane needs no clearing.
inline int64_t conv_state_elems(const ConvDims& m) { return m.taps > 1 ? (m.taps - 1) * m.channels : 0; }

struct ConvArgs {
  ConvDims m;
  const float* partial;    // first channel of the projection's slabs [nsplit][rows][ld]
  int nsplit;
  int64_t split_stride, ld;
  RowMap map;
  int capacity;            // positions a lane can have
  void* out;               // act dtype: [rows][ldo], or (group > 0) [channels / group][rows][ldo]
  int64_t ldo;
  int group;
  int* offsets;            // group > 0: gets the first row of every group, and the end
  int dtype;
  float* state;            // [lanes][taps - 1][channels]
  const int2* tails;       // rows whose inputs enter the state (see GqaPostArgs), nullptr: every row of a step of single tokens
  int n_tails;
  int early;               // captured decode step: state and positions predate the step
  int* status;
};
int conv_launch(Ctx* c, const ConvArgs& a, int64_t rows);   // and the state

}  // namespace rewb
