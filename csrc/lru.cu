// Gated linear recurrence of one value per channel (models/deluvik.py):
//
//   r = sigmoid(R u + b_r), i = sigmoid(I u + b_i)      R, I block-diagonal, u the convolved branch
//   log a = -8 r softplus(lam),  S_t = a S_(t-1) + sqrt(1 - a^2) i u,  out = S_t gelu(y) factor
//
//   lru_scan_kernel   gate pre-activations given (library product): 32 (16) channels of a sequence per block, 128 (256) tokens at a
//                     time; runs of 8 tokens are scanned from zero, the carries meet in shared memory.  Any length, verify windows
//                     (a state plane per token) included.
//   lru_step_kernel   one token per sequence (decode ticks): convolution, gates (mma.sync in bf16) and recurrence in one launch; a
//                     block owns 16 or 64 channels and streams their rows of R and I once for up to 8 sequences.
//
// Everything behind u is fp32.
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

constexpr float LRU_LOG2E = 1.4426950408889634f;
__device__ __forceinline__ float lru_ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float lru_sigmoid(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(1.f + lru_ex2(-LRU_LOG2E * x)));
  return y;
}
// the tanh form of gelu: z / 2 (1 + tanh(t)) = z sigmoid(2 t)
__device__ __forceinline__ float lru_gelu(float z) { return z * lru_sigmoid(1.5957691216057308f * (z + 0.044715f * z * z * z)); }
// (a, input factor) of the recurrence from the gates' pre-activations; sp: softplus(lam)
__device__ __forceinline__ float2 lru_decay(float zr, float zi, float sp) {
  const float la = -8.f * lru_sigmoid(zr) * sp, a = lru_ex2(LRU_LOG2E * la), t = 2.f * la;
  // 1 - a^2 = 1 - e^t; near t = 0 by the exponential series, whose first omitted term is t^6 / 5040 of the sum
  const float near = -t * fmaf(t * (1.f / 2.f), fmaf(t * (1.f / 3.f), fmaf(t * (1.f / 4.f), fmaf(t * (1.f / 5.f), fmaf(t, 1.f / 6.f, 1.f), 1.f), 1.f), 1.f), 1.f);
  const float left = t > -0.25f ? near : fmaf(-a, a, 1.f);
  float root;
  asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(root) : "f"(left));
  return make_float2(a, root * lru_sigmoid(zi));
}

// CH channels a block; a warp holds 32 / CH runs of LS_L consecutive tokens, one channel a lane.
constexpr int LS_WARPS = 16, LS_L = 8;
template <typename T, int CH>
__global__ void __launch_bounds__(LS_WARPS * 32) lru_scan_kernel(const LruArgs a) {
  constexpr int RUNS = LS_WARPS * (32 / CH), TILE = RUNS * LS_L;
  __shared__ float s_a[2][RUNS][CH], s_s[2][RUNS][CH];
  pdl_launch_dependents(54);
  pdl_wait();
  const int lane = threadIdx.x % CH, run = threadIdx.x / CH, seq = blockIdx.y, ch = blockIdx.x * CH + lane;
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
  float zr[LS_L], zi[LS_L];
  T uu[LS_L], yy[LS_L];
  auto load = [&](int f) {                                          // (tokens past the end repeat the last one: never used)
#pragma unroll
    for (int k = 0; k < LS_L; ++k) {
      const int t = min(f + k, n - 1);
      zr[k] = z[(size_t)t * 2 * a.pp], zi[k] = z[(size_t)t * 2 * a.pp + a.pp];
      uu[k] = u[(size_t)t * a.width], yy[k] = y[(size_t)t * a.ldp];
    }
  };
  load(run * LS_L);
  int buf = 0;
  for (int i0 = 0; i0 < n; i0 += TILE, buf ^= 1) {
    const int f = i0 + run * LS_L, m = n - f;                       // this run's first token; tokens left (<= 0: none)
    float pa[LS_L], ps[LS_L], g[LS_L];                              // product of decays and state from zero up to each token
    float A = 1.f, S = 0.f;
#pragma unroll
    for (int k = 0; k < LS_L; ++k) {
      const float2 d = lru_decay(zr[k] + br, zi[k] + bi, sp);
      if (k < m) A *= d.x, S = fmaf(d.x, S, d.y * to_f(uu[k]));
      pa[k] = A, ps[k] = S;
      g[k] = lru_gelu(to_f(yy[k]) + yb) * a.factor;
    }
    s_a[buf][run][lane] = A, s_s[buf][run][lane] = S;
    if (i0 + TILE < n) load(f + TILE);                              // the next tile's rows travel while the carries meet
    __syncthreads();
    float from = carry;
#pragma unroll
    for (int w = 0; w < RUNS; ++w) {
      if (w == run) from = carry;
      carry = fmaf(s_a[buf][w][lane], carry, s_s[buf][w][lane]);
    }
#pragma unroll
    for (int k = 0; k < LS_L; ++k) {
      if (k < m && in) {
        const float now = fmaf(pa[k], from, ps[k]);
        out[(size_t)(f + k) * a.ldo] = from_f<T>(now * g[k]);
        if (keep) rec[(size_t)(f + k) * a.plane_stride] = now;
      }
    }
  }
  if (!keep && run == 0 && in) rec[plane] = carry;
}

// grid (groups of CH channels within a part, groups of 8 sequences).  bf16: the gates' rows times the convolved rows on tensor cores,
// K split over the warps; fp32: two channels a warp at a time.
constexpr int LT_NB = 8, LT_PAD = 16;
template <typename T, int CH>
__global__ void __launch_bounds__(256) lru_step_kernel(const LruArgs a, int B) {
  constexpr int C = Chunk<T>::N;
  constexpr bool MMA = sizeof(T) == 2;
  extern __shared__ __align__(16) unsigned char lt_smem[];
  T* s_u = reinterpret_cast<T*>(lt_smem);                   // [8][ldu] convolved rows
  const int ldu = (a.pp + 31) / 32 * 32 + LT_PAD;
  float* s_z = reinterpret_cast<float*>(lt_smem + (size_t)LT_NB * ldu * sizeof(T));      // MMA: [8 warps][2][CH][8]; else [2][CH][8]
  pdl_launch_dependents(55);
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, groups = (a.pp + CH - 1) / CH;
  const int b = blockIdx.x / groups, g0 = (blockIdx.x % groups) * CH, m0 = blockIdx.y * LT_NB, nb = min(LT_NB, B - m0);
  const int chans = min(CH, a.pp - g0);
  pdl_wait();
  for (int x = tid; x < LT_NB * (ldu / C); x += 256) {
    const int m = x / (ldu / C), j = x % (ldu / C) * C, c = b * a.pp + j;
    float v[C];
#pragma unroll
    for (int e = 0; e < C; ++e) v[e] = 0.f;
    if (m < nb && j < a.pp) {
      const int t = a.q_start[m0 + m], pos = a.positions[t];
      T* rg = reinterpret_cast<T*>(a.ring) + (size_t)a.slots[m0 + m] * a.ring_slot + c;
      const uint4 own = *reinterpret_cast<const uint4*>(reinterpret_cast<const T*>(a.u) + (size_t)t * a.ldp + c);
#pragma unroll
      for (int e = 0; e < C; ++e) v[e] = a.conv_b[c + e];
      for (int back = 0; back < a.taps && back <= pos; ++back) {
        float f[C];
        Chunk<T>::get(back ? *reinterpret_cast<const uint4*>(rg + (size_t)((pos - back) % a.ring_rows) * a.ring_ld) : own, f);
#pragma unroll
        for (int e = 0; e < C; ++e) v[e] = fmaf(f[e] + a.x_b[c + e], a.conv[(size_t)(a.taps - 1 - back) * a.width + c + e], v[e]);
      }
      if (j >= g0 && j < g0 + CH) *reinterpret_cast<uint4*>(rg + (size_t)(pos % a.ring_rows) * a.ring_ld) = own;
    }
    *reinterpret_cast<uint4*>(s_u + (size_t)m * ldu + j) = Chunk<T>::put(v);
  }
  __syncthreads();
  const T* wg = reinterpret_cast<const T*>(a.gates) + ((size_t)b * 2 * a.pp + g0) * a.pp;
  if constexpr (MMA) {
    // a lane feeds 8 consecutive k of rows g and g + 8 to two MMAs under a permutation of k that both operands share
    const int g = lane >> 2, t = lane & 3;
    float acc[2 * (CH / 16)][4];
#pragma unroll
    for (int i = 0; i < 2 * (CH / 16); ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    for (int k0 = warp * 32; k0 < a.pp; k0 += 8 * 32) {
      const int k = k0 + t * 8;
      const uint4 xv = *reinterpret_cast<const uint4*>(s_u + (size_t)g * ldu + k);
#pragma unroll
      for (int i = 0; i < 2 * (CH / 16); ++i) {
        const int r = (i & 1) * a.pp + (i >> 1) * 16 + g;            // row of the recurrence gate, then of the input gate
        uint4 va = make_uint4(0u, 0u, 0u, 0u), vb = va;
        if (k < a.pp && (i >> 1) * 16 < chans) {
          va = ldg_stream_16(wg + (size_t)r * a.pp + k);
          vb = ldg_stream_16(wg + (size_t)(r + 8) * a.pp + k);
        }
        const uint32_t a0[4] = {va.x, vb.x, va.y, vb.y}, a1[4] = {va.z, vb.z, va.w, vb.w};
        mma16(acc[i], a0, xv.x, xv.y);
        mma16(acc[i], a1, xv.z, xv.w);
      }
    }
    // accumulator e: channel g + 8 (e / 2) of its tile, sequence 2 t + e % 2
#pragma unroll
    for (int i = 0; i < 2 * (CH / 16); ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e) s_z[((warp * 2 + (i & 1)) * CH + (i >> 1) * 16 + g + (e >> 1) * 8) * LT_NB + 2 * t + (e & 1)] = acc[i][e];
  } else {
    for (int i = warp; i < 2 * chans; i += 8) {
      const int gate = i / chans, j = i % chans;
      const T* w = wg + ((size_t)gate * a.pp + j) * a.pp;
      float acc[LT_NB];
#pragma unroll
      for (int m = 0; m < LT_NB; ++m) acc[m] = 0.f;
      for (int k = lane; k < a.pp; k += 32) {
        const float f = to_f(w[k]);
#pragma unroll
        for (int m = 0; m < LT_NB; ++m) acc[m] = fmaf(f, to_f(s_u[(size_t)m * ldu + k]), acc[m]);
      }
#pragma unroll
      for (int m = 0; m < LT_NB; ++m) {
        const float v = warp_sum(acc[m]);
        if (lane == 0) s_z[(gate * CH + j) * LT_NB + m] = v;
      }
    }
  }
  __syncthreads();
  for (int x = tid; x < chans * nb; x += 256) {
    const int m = x / chans, j = x % chans, c = b * a.pp + g0 + j, seq = m0 + m, t = a.q_start[seq], slot = a.slots[seq];
    float zr = 0.f, zi = 0.f;
#pragma unroll
    for (int k = 0; k < (MMA ? 8 : 1); ++k) zr += s_z[((k * 2) * CH + j) * LT_NB + m], zi += s_z[((k * 2 + 1) * CH + j) * LT_NB + m];
    float* st = a.states + (size_t)slot * a.slot_stride + (size_t)a.cur[slot] * a.plane_stride + c;
    const size_t gb = (size_t)b * 2 * a.pp + g0 + j;
    const float2 d = lru_decay(zr + a.gates_b[gb], zi + a.gates_b[gb + a.pp], softplus_x(a.lam[c]));
    const float S = fmaf(d.x, *st, d.y * to_f(s_u[(size_t)m * ldu + g0 + j]));
    *st = S;
    const float yv = to_f(reinterpret_cast<const T*>(a.y)[(size_t)t * a.ldp + c]) + a.y_b[c];
    reinterpret_cast<T*>(a.out)[(size_t)t * a.ldo + c] = from_f<T>(S * lru_gelu(yv) * a.factor);
  }
}

template <typename T, int CH>
cudaError_t step_launch(const LruArgs& a, int B, cudaStream_t st) {
  auto k = lru_step_kernel<T, CH>;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return e;
    configured = true;
  }
  const size_t smem = (size_t)LT_NB * ((a.pp + 31) / 32 * 32 + LT_PAD) * sizeof(T) + (size_t)(sizeof(T) == 2 ? 8 : 1) * 2 * CH * LT_NB * sizeof(float);
  if (smem > 200 * 1024) return cudaErrorInvalidValue;
  return trl_launch(k, dim3(a.width / a.pp * ((a.pp + CH - 1) / CH), (B + LT_NB - 1) / LT_NB), dim3(256), smem, st, a, B);
}

bool lru_bad(const LruArgs& a) {
  return a.width <= 0 || a.pp <= 0 || a.pp % 16 || a.width % a.pp || a.T <= 0 || !a.y || !a.u || !a.y_b || !a.gates_b || !a.lam || !a.states ||
         !a.cur || !a.out;
}

}  // namespace

TRL_API int trl_lru_scan(const LruArgs* a, int B, int f32, void* stream) {
  if (B <= 0 || lru_bad(*a) || !a->z) return (int)cudaErrorInvalidValue;
  cudaStream_t st = (cudaStream_t)stream;
  const bool narrow = (a->width + 31) / 32 * B < 128;             // too few blocks of 32 channels to fill the GPU
  const dim3 grid((a->width + (narrow ? 15 : 31)) / (narrow ? 16 : 32), B), thr(LS_WARPS * 32);
  if (f32) return (int)trl_launch(lru_scan_kernel<float, 32>, dim3((a->width + 31) / 32, B), thr, 0, st, *a);
  if (narrow) return (int)trl_launch(lru_scan_kernel<bf16, 16>, grid, thr, 0, st, *a);
  return (int)trl_launch(lru_scan_kernel<bf16, 32>, grid, thr, 0, st, *a);
}

// Every sequence of the batch has one token.
TRL_API int trl_lru_step(const LruArgs* a, int B, int f32, void* stream) {
  const int per = f32 ? 4 : 8;
  if (B <= 0 || lru_bad(*a) || !a->gates || !a->conv || !a->conv_b || !a->x_b || !a->ring || a->taps < 1 || a->taps > a->ring_rows ||
      a->ldp % per || a->ring_ld % per || a->ring_slot % per || ((uintptr_t)a->gates & 15) || ((uintptr_t)a->u & 15) || ((uintptr_t)a->ring & 15))
    return (int)cudaErrorInvalidValue;
  cudaStream_t st = (cudaStream_t)stream;
  if (f32) return (int)step_launch<float, 16>(*a, B, st);
  return (int)(B > LT_NB ? step_launch<bf16, 64>(*a, B, st) : step_launch<bf16, 16>(*a, B, st));
}
