// Gated linear recurrence of one value per channel (models/deluvik.py):
//
//   r = sigmoid(R u + b_r), i = sigmoid(I u + b_i)      R, I block-diagonal, u the convolved branch
//   log a = -8 r softplus(lam),  S_t = a S_(t-1) + sqrt(1 - a^2) i u,  out = S_t gelu(y) factor
//
//   lru_scan_kernel   gate pre-activations given (library product): 32 channels of a sequence per block, 128 tokens at a time; a
//                     warp scans 16 of them from zero, the carries meet in shared memory.  Any length, verify windows (a state
//                     plane per token) included.
//   lru_step_kernel   one token per sequence (decode ticks): convolution, gates and recurrence in one launch; a block owns 16
//                     channels and streams their rows of R and I once for up to 8 sequences.
//
// Everything behind u is fp32; sqrt(1 - a^2) is formed from expm1 of the exponent.
// Reference parity: the reference's recurrence is Gated DeltaNet only (no counterpart).
#include "packed.cuh"

// Mirrored by tilerl_b200/ops/cuda_blocks.py::LruArgs, field by field.
struct LruArgs {
  const void* y;                       // [T, ldp] gelu branch of the fused projection rows
  const float* y_b;
  const void* u;                       // scan: [T, width] convolved; step: [T, ldp] projected, not convolved
  const float* z;                      // scan: [blocks, T, 2 pp] products of both gates
  const float *gates_b, *lam;          // [blocks, 2 pp], [width]
  const void* gates;                   // step: [blocks, 2 pp, pp]
  const float *conv, *conv_b, *x_b;    // step: [taps, width], [width], [width]
  void* ring;                          // step: the layer's first column of slot 0
  long ring_slot;
  float* states;                       // the layer's record of slot 0, plane 0
  long slot_stride, plane_stride;      // floats
  const int *cur, *keep_flags, *q_start, *q_len, *slots, *positions;
  void* out;                           // first column of the result
  int ldp, ldo, T, width, pp, taps, ring_rows, ring_ld;
  float factor;
};

namespace {

// (a, input factor) of the recurrence from the gates' pre-activations
__device__ __forceinline__ float2 lru_decay(float zr, float zi, float sp) {
  const float la = -8.f * sigmoid_x(zr) * sp;
  return make_float2(expf(la), sqrtf(-expm1f(2.f * la)) * sigmoid_x(zi));
}

constexpr int LS_WARPS = 8, LS_L = 16, LS_TILE = LS_WARPS * LS_L;
template <typename T>
__global__ void __launch_bounds__(LS_WARPS * 32) lru_scan_kernel(const LruArgs a) {
  __shared__ float s_a[2][LS_WARPS][32], s_s[2][LS_WARPS][32];
  pdl_launch_dependents(54);
  pdl_wait();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, seq = blockIdx.y, ch = blockIdx.x * 32 + lane;
  const int n = a.q_len[seq], t0 = a.q_start[seq], slot = a.slots[seq];
  if (n <= 0) return;
  const bool in = ch < a.width, keep = a.keep_flags && a.keep_flags[seq];
  const int c = in ? ch : 0, b = c / a.pp, j = c % a.pp;
  float* rec = a.states + (size_t)slot * a.slot_stride + c;
  const size_t plane = (size_t)a.cur[slot] * a.plane_stride;
  const float sp = softplus_x(a.lam[c]), br = a.gates_b[(size_t)b * 2 * a.pp + j], bi = a.gates_b[(size_t)b * 2 * a.pp + a.pp + j], yb = a.y_b[c];
  const float* z = a.z + ((size_t)b * a.T + t0) * 2 * a.pp + j;
  const T* u = reinterpret_cast<const T*>(a.u) + (size_t)t0 * a.width + c;
  const T* y = reinterpret_cast<const T*>(a.y) + (size_t)t0 * a.ldp + c;
  T* out = reinterpret_cast<T*>(a.out) + (size_t)t0 * a.ldo + c;
  float carry = rec[plane];
  int buf = 0;
  for (int i0 = 0; i0 < n; i0 += LS_TILE, buf ^= 1) {
    const int f = i0 + warp * LS_L, m = min(LS_L, n - f);          // this warp's tokens (m <= 0: none)
    float pa[LS_L], ps[LS_L];                                       // product of decays and state from zero, up to each token
    {
      float zr[LS_L], zi[LS_L], uu[LS_L];
#pragma unroll
      for (int k = 0; k < LS_L; ++k) {
        const bool ok = k < m;
        zr[k] = ok ? z[(size_t)(f + k) * 2 * a.pp] : 0.f;
        zi[k] = ok ? z[(size_t)(f + k) * 2 * a.pp + a.pp] : 0.f;
        uu[k] = ok ? to_f(u[(size_t)(f + k) * a.width]) : 0.f;
      }
      float A = 1.f, S = 0.f;
#pragma unroll
      for (int k = 0; k < LS_L; ++k) {
        if (k < m) {
          const float2 d = lru_decay(zr[k] + br, zi[k] + bi, sp);
          A *= d.x, S = fmaf(d.x, S, d.y * uu[k]);
        }
        pa[k] = A, ps[k] = S;
      }
    }
    s_a[buf][warp][lane] = pa[LS_L - 1], s_s[buf][warp][lane] = ps[LS_L - 1];
    __syncthreads();
    float from = carry;
#pragma unroll
    for (int w = 0; w < LS_WARPS; ++w) {
      if (w == warp) from = carry;
      carry = fmaf(s_a[buf][w][lane], carry, s_s[buf][w][lane]);
    }
#pragma unroll
    for (int k = 0; k < LS_L; ++k) {
      if (k < m && in) {
        const float S = fmaf(pa[k], from, ps[k]);
        out[(size_t)(f + k) * a.ldo] = from_f<T>(S * gelu_tanh_x(to_f(y[(size_t)(f + k) * a.ldp]) + yb) * a.factor);
        if (keep) rec[(size_t)(f + k) * a.plane_stride] = S;
      }
    }
  }
  if (!keep && warp == 0 && in) rec[plane] = carry;
}

// grid (channel groups of 16 within a part, groups of NB sequences), 8 warps of two channels each
constexpr int LT_CH = 16;
template <typename T, int NB>
__global__ void __launch_bounds__(256) lru_step_kernel(const LruArgs a, int B) {
  constexpr int C = Chunk<T>::N;
  extern __shared__ __align__(16) float s_u[];              // [NB][pp]
  pdl_launch_dependents(55);
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, groups = a.pp / LT_CH;
  const int b = blockIdx.x / groups, g0 = (blockIdx.x % groups) * LT_CH, m0 = blockIdx.y * NB, nb = min(NB, B - m0);
  for (int x = tid; x < NB * a.pp; x += 256) {
    const int m = x / a.pp, j = x % a.pp, c = b * a.pp + j;
    float v = 0.f;
    if (m < nb) {
      const int t = a.q_start[m0 + m], pos = a.positions[t];
      T* rg = reinterpret_cast<T*>(a.ring) + (size_t)a.slots[m0 + m] * a.ring_slot + c;
      const T own = reinterpret_cast<const T*>(a.u)[(size_t)t * a.ldp + c];
      v = fmaf(to_f(own) + a.x_b[c], a.conv[(size_t)(a.taps - 1) * a.width + c], a.conv_b[c]);
      for (int back = 1; back < a.taps && back <= pos; ++back)
        v = fmaf(to_f(rg[(size_t)((pos - back) % a.ring_rows) * a.ring_ld]) + a.x_b[c], a.conv[(size_t)(a.taps - 1 - back) * a.width + c], v);
      v = to_f(from_f<T>(v));
      if (j >= g0 && j < g0 + LT_CH) rg[(size_t)(pos % a.ring_rows) * a.ring_ld] = own;
    }
    s_u[x] = v;
  }
  __syncthreads();
#pragma unroll
  for (int i = 0; i < LT_CH / 8; ++i) {
    const int j = g0 + warp * (LT_CH / 8) + i, c = b * a.pp + j;
    const T* wr = reinterpret_cast<const T*>(a.gates) + ((size_t)b * 2 * a.pp + j) * a.pp;
    const T* wi = wr + (size_t)a.pp * a.pp;
    float zr[NB], zi[NB];
#pragma unroll
    for (int m = 0; m < NB; ++m) zr[m] = zi[m] = 0.f;
    for (int k = lane * C; k < a.pp; k += 32 * C) {
      float fr[C], fi[C];
      Chunk<T>::get(*reinterpret_cast<const uint4*>(wr + k), fr);
      Chunk<T>::get(*reinterpret_cast<const uint4*>(wi + k), fi);
#pragma unroll
      for (int m = 0; m < NB; ++m)
#pragma unroll
        for (int e = 0; e < C; ++e) {
          const float v = s_u[m * a.pp + k + e];
          zr[m] = fmaf(fr[e], v, zr[m]), zi[m] = fmaf(fi[e], v, zi[m]);
        }
    }
    float r = 0.f, q = 0.f;                                  // lane m: the sums of sequence m
#pragma unroll
    for (int m = 0; m < NB; ++m) {
      const float sr = warp_sum(zr[m]), si = warp_sum(zi[m]);
      if (lane == m) r = sr, q = si;
    }
    if (lane < nb) {
      const int seq = m0 + lane, t = a.q_start[seq], slot = a.slots[seq];
      float* st = a.states + (size_t)slot * a.slot_stride + (size_t)a.cur[slot] * a.plane_stride + c;
      const float2 d = lru_decay(r + a.gates_b[(size_t)b * 2 * a.pp + j], q + a.gates_b[(size_t)b * 2 * a.pp + a.pp + j], softplus_x(a.lam[c]));
      const float S = fmaf(d.x, *st, d.y * s_u[lane * a.pp + j]);
      *st = S;
      const float yv = to_f(reinterpret_cast<const T*>(a.y)[(size_t)t * a.ldp + c]) + a.y_b[c];
      reinterpret_cast<T*>(a.out)[(size_t)t * a.ldo + c] = from_f<T>(S * gelu_tanh_x(yv) * a.factor);
    }
  }
}

template <typename T>
cudaError_t step_launch(const LruArgs& a, int B, cudaStream_t st) {
#define LRU_STEP(NB)                                                                                                       \
  {                                                                                                                        \
    auto k = lru_step_kernel<T, NB>;                                                                                       \
    static bool configured = false;                                                                                        \
    if (!configured) {                                                                                                     \
      const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);              \
      if (e != cudaSuccess) return e;                                                                                      \
      configured = true;                                                                                                   \
    }                                                                                                                      \
    return trl_launch(k, dim3(a.width / LT_CH, (B + NB - 1) / NB), dim3(256), (size_t)NB * a.pp * sizeof(float), st, a, B); \
  }
  if (B == 1) LRU_STEP(1)
  if (B == 2) LRU_STEP(2)
  if (B <= 4 || a.pp > 4096) LRU_STEP(4)
  LRU_STEP(8)
#undef LRU_STEP
}

bool lru_bad(const LruArgs& a) {
  return a.width <= 0 || a.pp <= 0 || a.pp % 16 || a.width % a.pp || a.T <= 0 || !a.y || !a.u || !a.y_b || !a.gates_b || !a.lam || !a.states ||
         !a.cur || !a.out;
}

}  // namespace

TRL_API int trl_lru_scan(const LruArgs* a, int B, int f32, void* stream) {
  if (B <= 0 || lru_bad(*a) || !a->z) return (int)cudaErrorInvalidValue;
  const dim3 grid((a->width + 31) / 32, B);
  if (f32) return (int)trl_launch(lru_scan_kernel<float>, grid, dim3(LS_WARPS * 32), 0, (cudaStream_t)stream, *a);
  return (int)trl_launch(lru_scan_kernel<bf16>, grid, dim3(LS_WARPS * 32), 0, (cudaStream_t)stream, *a);
}

// Every sequence of the batch has one token.
TRL_API int trl_lru_step(const LruArgs* a, int B, int f32, void* stream) {
  if (B <= 0 || lru_bad(*a) || !a->gates || !a->conv || !a->conv_b || !a->x_b || !a->ring || a->taps < 1 || a->taps > a->ring_rows ||
      a->pp > 8192 || ((uintptr_t)a->gates & 15))
    return (int)cudaErrorInvalidValue;
  return (int)(f32 ? step_launch<float>(*a, B, (cudaStream_t)stream) : step_launch<bf16>(*a, B, (cudaStream_t)stream));
}
