// What the expert kernels share (moe.cu, moe_tc.cu).
#pragma once
#include "packed.cuh"

// One tile of rows of an expert: rows [row0, row0 + n) of the list ordered by expert.
struct MoeItem {
  int expert, row0, n, pad;
};

// projections of the tiles: gated up (pairs of weight rows), down, plain up (an activation of every weight row)
enum { MOE_UP = 0, MOE_DOWN = 1, MOE_ACT = 2 };
