// Building device matrices from host tensors or from the seeded generator, shared by the model families.
#pragma once

#include <vector>

#include "pi_common.cuh"

namespace pi_load {

struct Source {
  const pi_tensor* host = nullptr;  // host tensor, or
  bool synthetic = false;           // device-generated N(0, std)
  uint64_t seed = 0, stream_id = 0;
  float std = 0.02f;
  int kind = PI_F32;                // synthetic: kind AFTER load (PI_INT8 or PI_BF16)
  size_t rows = 0, cols = 0;
};

// A local (per-rank) matrix whose rows are slices of one or more sources.
struct Piece {
  Source src;
  size_t src_r0, nrows;  // rows taken from the source
  size_t dst_r0, step;   // where they land
};

pi_status build_linear(pi_ctx* ctx, const std::vector<Piece>& pieces, size_t local_rows, size_t local_cols, size_t c0,
                       pi_linear** out);

}  // namespace pi_load
