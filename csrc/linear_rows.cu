// bf16 projections of 1..16 rows into or out of an fp32 residual stream (decode and small mixed ticks).
//
//   y[m, n] (store bf16 | store fp32 | += fp32) = sum_k x'[m, k] * W[n, k]
//
// x' is the row itself (bf16) or rms(x) * norm_w of an fp32 stream row, rounded to bf16.  The weights are
// streamed once, straight into mma.sync A fragments: a warp owns 16 weight rows and a share of K; lane (g, t)
// loads 16 bytes (8 consecutive k) of rows g and g + 8 per 32-wide step.  The order of k does not matter to a
// dot product, so the 8 values serve two MMAs under a fixed permutation of k that the activation chunk (read
// from shared memory as one 16-byte load) shares.  KW warps of a block split K and meet in shared memory in a
// fixed order, so a run repeats bit for bit.  A block stages the activations once and walks its row tiles, the next
// tile's first weights in flight while one is summed up.  The first weight loads are issued before the dependency wait:
// weights are constants of the tick.
// Reference parity: it projects out of a bf16 residual (no counterpart).
#include "common.cuh"

namespace {

constexpr int LR_THREADS = 256, LR_WARPS = LR_THREADS / 32, LR_U = 8, LR_PAD = 32;
constexpr int LR_SMEM = 160 * 1024;
enum { LR_STORE = 0, LR_STORE_F32 = 1, LR_ADD_F32 = 2 };

__device__ __forceinline__ void lr_mma(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

template <bool NORM, int NT, int EPI>
__global__ void __launch_bounds__(LR_THREADS, 2)
linear_rows_kernel(const void* xin, int ldx, const bf16* __restrict__ w, const float* __restrict__ norm_w, float eps, int n_norm,
                   void* y, int ldy, int M, int N, int K, int kseg, int KW, int n_tiles) {
  extern __shared__ __align__(16) unsigned char lr_smem[];
  __shared__ float red[32];
  __shared__ float s_r[16];
  __shared__ float s_part[LR_WARPS * 16 * NT * 8];
  bf16* xs = reinterpret_cast<bf16*>(lr_smem);                 // [M][kseg + LR_PAD]
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
  const int RW = LR_WARPS / KW, wr = warp / KW, wk = warp % KW;
  const int nseg = (K + kseg - 1) / kseg, ldxs = kseg + LR_PAD;
  const bf16 *wa, *wb;
  auto rows_of = [&](int tile) {
    const int r0 = (tile * RW + wr) * 16;
    wa = w + (size_t)min(r0 + g, N - 1) * K + (t << 3), wb = w + (size_t)min(r0 + g + 8, N - 1) * K + (t << 3);
  };
  // this warp's 32-wide steps of segment s
  int jb, je;
  auto range = [&](int s) {
    const int steps = min(kseg, K - s * kseg) >> 5, per = (steps + KW - 1) / KW;
    jb = min(steps, wk * per), je = min(steps, jb + per);
  };
  uint4 va[LR_U], vb[LR_U];
  auto load = [&](int s, int j0) {
#pragma unroll
    for (int u = 0; u < LR_U; ++u) {
      const int j = min(j0 + u, je - 1);
      const size_t o = (size_t)s * kseg + ((size_t)j << 5);
      va[u] = ldg_stream_16(wa + o), vb[u] = ldg_stream_16(wb + o);
    }
  };
  rows_of(blockIdx.x);
  range(0);
  if (jb < je) load(0, jb);
  pdl_launch_dependents(24);
  pdl_wait();
  if (NORM) {
    for (int m = 0; m < M; ++m) {
      const float4* xr = reinterpret_cast<const float4*>(reinterpret_cast<const float*>(xin) + (size_t)m * ldx);
      float ss = 0.f;
      for (int c = threadIdx.x; c < K / 4; c += LR_THREADS) {
        const float4 v = xr[c];
        ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
      }
      ss = block_sum(ss, red);
      if (threadIdx.x == 0) s_r[m] = 1.f / sqrtf(ss / (float)n_norm + eps);
    }
  }
  auto stage = [&](int s) {
    __syncthreads();                                           // s_r written; the previous segment is consumed
    const int kc = min(kseg, K - s * kseg);
    for (int m = 0; m < M; ++m) {
      bf16* dst = xs + (size_t)m * ldxs;
      if (NORM) {
        const float* xr = reinterpret_cast<const float*>(xin) + (size_t)m * ldx + s * kseg;
        const float* nw = norm_w + s * kseg;
        const float r = s_r[m];
        for (int c = threadIdx.x; c < kc / 4; c += LR_THREADS) {
          const float4 v = *reinterpret_cast<const float4*>(xr + 4 * c), q = *reinterpret_cast<const float4*>(nw + 4 * c);
          *reinterpret_cast<uint2*>(dst + 4 * c) =
              make_uint2(f2_to_bf162_bits(v.x * r * q.x, v.y * r * q.y), f2_to_bf162_bits(v.z * r * q.z, v.w * r * q.w));
        }
      } else {
        const bf16* xr = reinterpret_cast<const bf16*>(xin) + (size_t)m * ldx + s * kseg;
        for (int c = threadIdx.x; c < kc / 8; c += LR_THREADS)
          *reinterpret_cast<uint4*>(dst + 8 * c) = *reinterpret_cast<const uint4*>(xr + 8 * c);
      }
    }
    __syncthreads();
  };
  if (nseg == 1) stage(0);
  for (int tile = blockIdx.x; tile < n_tiles; tile += gridDim.x) {
    float acc[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    for (int s = 0; s < nseg; ++s) {
      if (nseg > 1) {
        stage(s);
        range(s);
        if ((s > 0 || tile != blockIdx.x) && jb < je) load(s, jb);
      }
      for (int j0 = jb; j0 < je; j0 += LR_U) {
        if (j0 > jb) load(s, j0);
#pragma unroll
        for (int u = 0; u < LR_U; ++u) {
          if (j0 + u < je) {
#pragma unroll
            for (int i = 0; i < NT; ++i) {
              uint4 xv = make_uint4(0u, 0u, 0u, 0u);           // rows past M count as zeros
              if (i * 8 + g < M) xv = *reinterpret_cast<const uint4*>(xs + (size_t)(i * 8 + g) * ldxs + ((j0 + u) << 5) + (t << 3));
              lr_mma(acc[i], va[u].x, vb[u].x, va[u].y, vb[u].y, xv.x, xv.y);
              lr_mma(acc[i], va[u].z, vb[u].z, va[u].w, vb[u].w, xv.z, xv.w);
            }
          }
        }
      }
    }
    const int next = tile + gridDim.x;
    if (next < n_tiles) {
      rows_of(next);
      if (nseg == 1 && jb < je) load(0, jb);                   // in flight while this tile is summed up
    }
    // accumulator e of tile i: weight row g + 8 (e / 2), activation row 8 i + 2 t + e % 2
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e)
        s_part[(warp * NT * 8 + i * 8 + 2 * t + (e & 1)) * 16 + g + (e >> 1) * 8] = acc[i][e];
    __syncthreads();
    for (int x = threadIdx.x; x < RW * 16 * M; x += LR_THREADS) {
      const int m = x / (RW * 16), c = x % (RW * 16), n = tile * RW * 16 + c;
      if (n >= N) continue;
      float v = 0.f;
      for (int k = 0; k < KW; ++k) v += s_part[(((c >> 4) * KW + k) * NT * 8 + m) * 16 + (c & 15)];
      if (EPI == LR_STORE) reinterpret_cast<bf16*>(y)[(size_t)m * ldy + n] = __float2bfloat16(v);
      else if (EPI == LR_STORE_F32) reinterpret_cast<float*>(y)[(size_t)m * ldy + n] = v;
      else reinterpret_cast<float*>(y)[(size_t)m * ldy + n] += v;
    }
    __syncthreads();
  }
}

int lr_sms() {
  static int n = [] {
    int dev = 0, v = 148;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&v, cudaDevAttrMultiProcessorCount, dev);
    return v;
  }();
  return n;
}

}  // namespace

// x: bf16 [M, ldx], or the fp32 stream when norm_w is given (its row norm counts n_norm columns).  w: bf16 [N, K],
// K a multiple of 64.  epi: 0 store bf16, 1 store fp32, 2 add to fp32.  M <= 16.
TRL_API int trl_linear_rows(const void* x, int ldx, const void* w, const void* norm_w, float eps, int n_norm, void* y, int ldy,
                            int M, int N, int K, int epi, void* stream) {
  if (M < 1 || M > 16 || N < 1 || K < 64 || K % 64 || ldx % 8 || epi < 0 || epi > 2 || (norm_w && n_norm < 1) ||
      ((uintptr_t)x & 15) || ((uintptr_t)w & 15))
    return (int)cudaErrorInvalidValue;
  const int groups = (N + 15) / 16;
  // split K over the warps of a block: shares of at least 16 steps, more splits where there are few rows
  int KW = 1;
  while (KW < LR_WARPS && (K / 32 / (2 * KW) >= 16 || (long)groups * KW < 2L * lr_sms() * LR_WARPS)) KW *= 2;
  const int RW = LR_WARPS / KW, n_tiles = (groups + RW - 1) / RW;
  const int cap = (LR_SMEM / (2 * M) - LR_PAD) / 32 * 32;
  const int nseg = (K + cap - 1) / cap, kseg = ((K + nseg - 1) / nseg + 31) / 32 * 32;
  const size_t smem = (size_t)M * (kseg + LR_PAD) * sizeof(bf16);
  const int nt = M <= 8 ? 1 : 2;
  const int grid = min(n_tiles, lr_sms() * (smem <= 96 * 1024 ? 2 : 1));   // one round of blocks walks all row tiles
  cudaError_t e = cudaErrorInvalidValue;
#define LR_CASE(NO, NTT, EP)                                                                                            \
  if ((norm_w != nullptr) == NO && nt == NTT && epi == EP) {                                                            \
    auto kern = linear_rows_kernel<NO, NTT, EP>;                                                                        \
    static bool configured = false;                                                                                     \
    if (!configured) {                                                                                                  \
      e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, LR_SMEM + 4096);                      \
      if (e != cudaSuccess) return (int)e;                                                                              \
      configured = true;                                                                                                \
    }                                                                                                                   \
    e = trl_launch(kern, dim3(grid), dim3(LR_THREADS), smem, (cudaStream_t)stream, x, ldx, (const bf16*)w,              \
                   (const float*)norm_w, eps, n_norm, y, ldy, M, N, K, kseg, KW, n_tiles);                                       \
  }
  LR_CASE(true, 1, LR_STORE) LR_CASE(true, 1, LR_STORE_F32) LR_CASE(true, 2, LR_STORE) LR_CASE(true, 2, LR_STORE_F32)
  LR_CASE(false, 1, LR_STORE) LR_CASE(false, 1, LR_STORE_F32) LR_CASE(false, 1, LR_ADD_F32)
  LR_CASE(false, 2, LR_STORE) LR_CASE(false, 2, LR_STORE_F32) LR_CASE(false, 2, LR_ADD_F32)
#undef LR_CASE
  return (int)e;
}
