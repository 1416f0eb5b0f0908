// Which sequence (lane) and position every row of a step belongs to, and runs of rows that a kernel works on together.
#pragma once
#include "common.cuh"

namespace rewb {

// Explicit arrays (a step of unequal portions), or S consecutive tokens for every lane from b0 on, starting at the
// lane's position pos0[lane].
struct RowMap {
  const int* row_lane;
  const int* row_pos;
  const int* pos0;
  int b0, S;
};

// Runs of consecutive rows of one lane: an explicit list of (first row, rows), or (list == nullptr) the rows of
// every lane of a uniform step in pieces of `per_tile`.
struct RowTiles {
  const int2* list;
  int count;      // tiles
  int S;          // rows per lane (list == nullptr)
  int per_tile;   // rows per tile at most
};

#ifdef __CUDACC__
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

template <typename T> __device__ __forceinline__ float ldf(T v);
template <> __device__ __forceinline__ float ldf<float>(float v) { return v; }
template <> __device__ __forceinline__ float ldf<bf16>(bf16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T stf(float v);
template <> __device__ __forceinline__ float stf<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 stf<bf16>(float v) { return __float2bfloat16_rn(v); }
#endif

}  // namespace rewb
