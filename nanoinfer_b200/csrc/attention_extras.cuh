// What the attention kernels share of the options in AttnExtras (api.h).
#pragma once

#include "api.h"
#include "common.cuh"

namespace nib {

// How many of the blocks 0, 1, ... of `pool` positions lie wholly behind the window of the row at `pos` (block b is seen
// if its last position (b + 1) pool - 1 <= pos - window).
__host__ __device__ __forceinline__ int pooled_blocks_seen(int pos, int window, int pool) {
  const int behind = pos - window + 1;   // positions 0 .. behind - 1 have left the window
  return pool > 0 && behind > 0 ? behind / pool : 0;
}

// The factor of a gate per element on value d of head h of row t (1 where there is none).
__device__ __forceinline__ float element_gate(const AttnExtras& ex, int t, int h, int d) {
  if (ex.gate == nullptr || ex.gate_dim <= 0 || d >= ex.gate_dim) return 1.0f;
  return 1.0f / (1.0f + expf(-ex.gate[(size_t)t * ex.ldg + h * ex.gate_dim + d]));
}

// Pooled blocks need a window and a table of their own, and go with no option that reads a key's position.
__host__ inline bool bad_pool(const AttnExtras& ex, int window) {
  if (ex.gate_dim < 0 || ex.pool < 0) return true;
  return ex.pool > 0 && (window <= 0 || ex.pool_table == nullptr || ex.slopes != nullptr || ex.keep_first > 0 || ex.span > 0);
}

}  // namespace nib
