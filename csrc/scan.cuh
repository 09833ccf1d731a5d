// Arguments and gates of the decayed-scan kernels (scan.cu, scan_mma.cu).
#pragma once
#include "packed.cuh"

enum { SCAN_MAMBA2 = 0, SCAN_MLSTM = 1, SCAN_FIXED = 2 };

// Mirrored by tilerl_b200/ops/cuda_mixers.py::ScanArgs, field by field.
struct ScanArgs {
  const void* rows;                    // [T, ld]: q, k, v columns at q0, k0, v0
  const float* gates;                  // [T, ldg] raw gates: dt, or i then f
  const float *gate_b, *a_log, *skip;  // per head (gate_b: per gate; a_log of SCAN_FIXED: log of what a head keeps)
  float* states;                       // the layer's record of slot 0, plane 0
  const int *cur, *keep_flags, *q_start, *q_len, *slots;
  float* o;                            // [T, heads * dv]
  long slot_stride, plane_stride;      // floats
  int ld, q0, k0, v0, ldg;
  int heads, per, dk, dv;              // per: heads that share q and k
  int min_len, max_len;
  float cap, q_scale;
  // decode ticks of Mamba-2: rows are not convolved yet, scan_serial_kernel does it (taps 0: they are)
  int taps, channels, ring_rows, ring_ld;
  const float *conv_w, *conv_b;        // [taps, channels], [channels]
  const void* ring;                    // the layer's first column of slot 0
  long ring_slot;
  const int* positions;
};

inline bool scan_args_bad(const ScanArgs& a, int kind) {
  return a.heads <= 0 || a.per <= 0 || a.heads % a.per || a.dk <= 0 || a.dk % 16 || a.dk > 256 || a.dv <= 0 || a.dv % 16 ||
         !a.rows || !a.states || !a.o || kind < SCAN_MAMBA2 || kind > SCAN_FIXED || (kind != SCAN_MLSTM && !a.a_log) ||
         (kind != SCAN_FIXED && (!a.gates || !a.gate_b || a.ldg < a.heads * (kind + 1))) || (kind == SCAN_MAMBA2 && !a.skip) ||
         (kind == SCAN_MLSTM && !(a.cap > 0.f));
}

// Mamba-2, fixed: (keep, what the token adds) of a token and head.  mLSTM: (log forget gate, log input gate).
template <int KIND>
__device__ __forceinline__ void scan_gates(const ScanArgs& a, int t, int h, float& g0, float& g1) {
  if (KIND == SCAN_FIXED) {
    g0 = expf(a.a_log[h]), g1 = 1.f;
    return;
  }
  const float* row = a.gates + (size_t)t * a.ldg;
  if (KIND == SCAN_MAMBA2) {
    g1 = softplus_x(row[h] + a.gate_b[h]);
    g0 = expf(-expf(a.a_log[h]) * g1);
  } else {
    g1 = a.cap * tanhf((row[h] + a.gate_b[h]) / a.cap);
    g0 = -softplus_x(-a.cap * tanhf((row[a.heads + h] + a.gate_b[a.heads + h]) / a.cap));
  }
}
