// Arguments of the per-channel delta rule's kernels (delta.cu, delta_mma.cu).
#pragma once
#include "packed.cuh"

// Mirrored by tilerl_b200/ops/cuda_gated.py::DeltaArgs, field by field.
struct DeltaArgs {
  const void* rows;                    // [T, ldp] projection rows: q, k, v columns at 0, k0, v0, channels in all
  const float *conv_w;                 // [taps, channels]
  void* ring;                          // earlier rows: the layer's first column of slot 0
  const float *low;                    // [T, heads * dk] decays before bias and softplus
  const float *dt_bias, *a_log;        // [heads * dk], [heads]
  const float* gates;                  // [T, ldg] write gates before the sigmoid
  float *q, *k;                        // [T, kv_heads * dk] unit rows, q times q_scale
  void* v;                             // [T, heads * dv]
  float *keep;                         // [T, heads * dk] log of what a channel keeps; may be `low` itself
  float *beta;                         // [T, heads]
  float* states;                       // the layer's record of slot 0, plane 0: S [heads, dk, dv]
  const int *cur, *keep_flags, *q_start, *q_len, *slots, *positions, *seq_ids;
  float* o;                            // [T, heads * dv]
  float* chunk;                        // scratch of the chunked form
  long ring_slot, slot_stride, plane_stride;
  int ldp, ldg, k0, v0, channels, taps, ring_rows, ring_ld, write_ring, heads, kv_heads, dk, dv, min_len, max_len;
  float q_scale;
};

inline bool delta_args_bad(const DeltaArgs& a) {
  return a.heads <= 0 || a.kv_heads <= 0 || a.heads % a.kv_heads || a.dk <= 0 || a.dk % 16 || a.dk > 256 || a.dv <= 0 || a.dv % 16 || !a.q || !a.k ||
         !a.v || !a.keep || !a.beta || a.k0 != a.kv_heads * a.dk || a.v0 != 2 * a.k0 || a.channels != a.v0 + a.heads * a.dv;
}
