// Library-wide device state: the error word every bounded wait and bounds check reports to, the switch for
// programmatic dependent launch, and the launch timeline of -DTRL_TRACE builds.
// Reference parity: none of its kernels reports errors this way (no counterpart).
#include "common.cuh"

__device__ TrlError g_trl_error = {0, 0, 0, 0};
int g_trl_use_pdl = 1;
#ifdef TRL_TRACE
__device__ TrlTraceRec g_trl_trace[TRL_TRACE_CAP];
__device__ unsigned int g_trl_trace_n = 0;
__device__ unsigned int g_trl_trace_cur = 0;
__device__ unsigned long long g_trl_last_exit = 0;
#endif

TRL_API void trl_set_pdl(int on) { g_trl_use_pdl = on; }

TRL_API int trl_error_read(int* out4, int clear) {
  TrlError h;
  cudaError_t e = cudaMemcpyFromSymbol(&h, g_trl_error, sizeof(h));
  if (e != cudaSuccess) return (int)e;
  out4[0] = h.code, out4[1] = h.a, out4[2] = h.b, out4[3] = h.c;
  if (clear && h.code != 0) {
    TrlError z = {0, 0, 0, 0};
    cudaMemcpyToSymbol(g_trl_error, &z, sizeof(z));
  }
  return 0;
}

// Timeline records of the launches since the last reset (builds with -DTRL_TRACE; otherwise
// returns 0 records).  out: n x 16 uint64 {kind, entry, dependency wait done, exit, mark 0, mark 1,
// latest exit of any CTA of the launches before, unused, marks 2..9} in ns.
TRL_API int trl_trace_read(void* out, int cap, int reset) {
#ifdef TRL_TRACE
  unsigned int n = 0;
  if (cudaMemcpyFromSymbol(&n, g_trl_trace_n, sizeof(n)) != cudaSuccess) return -1;
  if ((int)n > cap) n = cap;
  if (n > TRL_TRACE_CAP) n = TRL_TRACE_CAP;
  if (n && cudaMemcpyFromSymbol(out, g_trl_trace, (size_t)n * sizeof(TrlTraceRec)) != cudaSuccess) return -1;
  if (reset) {
    const unsigned int z = 0;
    cudaMemcpyToSymbol(g_trl_trace_n, &z, sizeof(z));
  }
  return (int)n;
#else
  (void)out, (void)cap, (void)reset;
  return 0;
#endif
}
