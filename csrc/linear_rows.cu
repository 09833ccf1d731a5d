// bf16 projections of 1..16 rows into or out of an fp32 residual stream (decode and small mixed ticks).
//
//   y[m, n] (store bf16 | store fp32 | += fp32) = sum_k x'[m, k] * W[n, k]
//
// or, in the epilogue, rows n >= n_split stored in fp32 beside the bf16 ones (gates of a recurrence or of a branch, whose rows may read
// another input), the first rows through an activation, pairs of rows (gate, up)
// joined by a gated activation, the soft cap of logits, or gelu(y) times a token's side-embedding row.
// x' is the row itself (bf16) or rms(x) * norm_w of an fp32 stream row, rounded to bf16.  The weights are streamed
// once: a warp owns 16 weight rows and a share of K, and every lane copies the 16-byte pieces it will itself feed to
// mma.sync (8 consecutive k of rows g and g + 8 per 32-wide step) into its own slots of a shared-memory ring, so no
// barrier sits between the copies and the products, and the bytes in flight do not depend on how much of the SM's
// memory is left to L1 (register loads lost half their rate behind a kernel that takes all of it as shared memory).
// The order of k does not matter to a dot product, so the 8 values serve two MMAs under a fixed permutation of k that
// the activation chunk (one 16-byte load) shares.  KW warps of a block split K and meet in shared memory in a fixed
// order, so a run repeats bit for bit.  A block stages the activations once and walks its row tiles; the ring runs on
// across tiles, and its first fill is issued before the dependency wait: weights are constants of the tick.
// Reference parity: it projects out of a bf16 residual (no counterpart).
#include "packed.cuh"

namespace {

constexpr int LR_THREADS = 256, LR_WARPS = LR_THREADS / 32, LR_U = 4, LR_PAD = 32;
constexpr int LR_SLOT = LR_U * 2 * 512;                        // bytes of a ring stage of one warp
constexpr int LR_SMEM = 216 * 1024;
enum { LR_STORE = 0, LR_STORE_F32 = 1, LR_ADD_F32 = 2, LR_GLU = 3, LR_SIDE = 4 };
struct LrExtra {
  float* y2;                                                   // LR_STORE: fp32 rows n >= n_split
  int ldy2, n_split;
  int n_act;                                                   // LR_STORE: act (ACT_*) of rows n < n_act
  const bf16* x2;                                              // rows n >= n_x2 (a multiple of 16) read this input
  int n_x2;
  int act;                                                     // LR_GLU: GLU_*
  float limit;
  float cap;                                                   // LR_STORE_F32: cap tanh(y / cap) (0: y)
  const int* ids;                                              // LR_SIDE: side[id * ld_side + off + n] for n < dim, 0 past it
  const bf16* side;
  long ld_side;
  int off, dim, vocab;
};

__device__ __forceinline__ void lr_mma(float (&c)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

__device__ __forceinline__ void lr_copy(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ uint4 lr_lds(uint32_t a) {
  uint4 v;
  asm volatile("ld.shared.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "r"(a) : "memory");
  return v;
}

template <bool NORM, int NT, int EPI, int DEPTH>
__global__ void __launch_bounds__(LR_THREADS)
linear_rows_kernel(const void* xin, int ldx, const bf16* __restrict__ w, const float* __restrict__ norm_w, float eps, int n_norm,
                   void* y, int ldy, int M, int N, int K, int KW, int n_tiles, const LrExtra ex) {
  extern __shared__ __align__(16) unsigned char lr_smem[];
  __shared__ float red[32];
  __shared__ float s_r[16];
  __shared__ float s_part[LR_WARPS * 16 * NT * 8];
  bf16* xs = reinterpret_cast<bf16*>(lr_smem + LR_WARPS * DEPTH * LR_SLOT);     // [M][K + LR_PAD]
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, g = lane >> 2, t = lane & 3;
  const int RW = LR_WARPS / KW, wr = warp / KW, wk = warp % KW, ldxs = K + LR_PAD;
  const uint32_t ring = (uint32_t)__cvta_generic_to_shared(lr_smem) + warp * DEPTH * LR_SLOT + lane * 16;
  const int steps = K >> 5, per = (steps + KW - 1) / KW, jb = min(steps, wk * per), je = min(steps, jb + per);
  // fetch cursor: runs DEPTH - 1 blocks of LR_U steps ahead of the products, across row tiles
  int f_tile = blockIdx.x, f_j = jb, f_slot = 0;
  auto fetch = [&]() {
    if (f_tile < n_tiles && jb < je) {
      const int r0 = (f_tile * RW + wr) * 16;
      const bf16* wa = w + (size_t)min(r0 + g, N - 1) * K + (t << 3);
      const bf16* wb = w + (size_t)min(r0 + g + 8, N - 1) * K + (t << 3);
#pragma unroll
      for (int u = 0; u < LR_U; ++u) {
        if (f_j + u < je) {
          const size_t o = (size_t)(f_j + u) << 5;
          lr_copy(ring + f_slot * LR_SLOT + u * 1024, wa + o);
          lr_copy(ring + f_slot * LR_SLOT + u * 1024 + 512, wb + o);
        }
      }
      f_j += LR_U;
      if (f_j >= je) f_j = jb, f_tile += gridDim.x;
    }
    f_slot = f_slot + 1 == DEPTH ? 0 : f_slot + 1;
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
#pragma unroll
  for (int i = 0; i < DEPTH - 1; ++i) fetch();
  pdl_enter(24);
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
    __syncthreads();
  }
  for (int m = 0; m < M; ++m) {
    bf16* dst = xs + (size_t)m * ldxs;
    if (NORM) {
      const float* xr = reinterpret_cast<const float*>(xin) + (size_t)m * ldx;
      const float r = s_r[m];
      for (int c = threadIdx.x; c < K / 4; c += LR_THREADS) {
        const float4 v = *reinterpret_cast<const float4*>(xr + 4 * c), q = *reinterpret_cast<const float4*>(norm_w + 4 * c);
        *reinterpret_cast<uint2*>(dst + 4 * c) =
            make_uint2(f2_to_bf162_bits(v.x * r * q.x, v.y * r * q.y), f2_to_bf162_bits(v.z * r * q.z, v.w * r * q.w));
      }
    } else {
      const bf16* xr = reinterpret_cast<const bf16*>(xin) + (size_t)m * ldx;
      for (int c = threadIdx.x; c < K / 8; c += LR_THREADS)
        *reinterpret_cast<uint4*>(dst + 8 * c) = *reinterpret_cast<const uint4*>(xr + 8 * c);
    }
  }
  if (EPI == LR_STORE && ex.x2)
    for (int m = 0; m < M; ++m)
      for (int c = threadIdx.x; c < K / 8; c += LR_THREADS)
        *reinterpret_cast<uint4*>(xs + (size_t)(M + m) * ldxs + 8 * c) = *reinterpret_cast<const uint4*>(ex.x2 + (size_t)m * ldx + 8 * c);
  __syncthreads();
  int slot = 0;
  for (int tile = blockIdx.x; tile < n_tiles; tile += gridDim.x) {
    const bf16* xt = EPI == LR_STORE && ex.x2 && (tile * RW + wr) * 16 >= ex.n_x2 ? xs + (size_t)M * ldxs : xs;
    if (tile + (int)gridDim.x >= n_tiles) pdl_trigger();       // last tile: dependents may take the room this block leaves
    float acc[NT][4];
#pragma unroll
    for (int i = 0; i < NT; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    for (int j0 = jb; j0 < je; j0 += LR_U) {
      fetch();
      asm volatile("cp.async.wait_group %0;" ::"n"(DEPTH - 1) : "memory");
      uint4 va[LR_U], vb[LR_U];
#pragma unroll
      for (int u = 0; u < LR_U; ++u) {
        va[u] = lr_lds(ring + slot * LR_SLOT + u * 1024);
        vb[u] = lr_lds(ring + slot * LR_SLOT + u * 1024 + 512);
      }
      slot = slot + 1 == DEPTH ? 0 : slot + 1;
#pragma unroll
      for (int u = 0; u < LR_U; ++u) {
        if (j0 + u < je) {
#pragma unroll
          for (int i = 0; i < NT; ++i) {
            uint4 xv = make_uint4(0u, 0u, 0u, 0u);             // rows past M count as zeros
            if (i * 8 + g < M) xv = *reinterpret_cast<const uint4*>(xt + (size_t)(i * 8 + g) * ldxs + ((j0 + u) << 5) + (t << 3));
            lr_mma(acc[i], va[u].x, vb[u].x, va[u].y, vb[u].y, xv.x, xv.y);
            lr_mma(acc[i], va[u].z, vb[u].z, va[u].w, vb[u].w, xv.z, xv.w);
          }
        }
      }
    }
    // accumulator e of tile i: weight row g + 8 (e / 2), activation row 8 i + 2 t + e % 2
#pragma unroll
    for (int i = 0; i < NT; ++i)
#pragma unroll
      for (int e = 0; e < 4; ++e)
        s_part[(warp * NT * 8 + i * 8 + 2 * t + (e & 1)) * 16 + g + (e >> 1) * 8] = acc[i][e];
    __syncthreads();
    auto total = [&](int m, int c) {
      float v = 0.f;
      for (int k = 0; k < KW; ++k) v += s_part[(((c >> 4) * KW + k) * NT * 8 + m) * 16 + (c & 15)];
      return v;
    };
    constexpr int PER = EPI == LR_GLU ? 8 : 16;                // outputs of a row tile
    for (int x = threadIdx.x; x < RW * PER * M; x += LR_THREADS) {
      const int m = x / (RW * PER), c = x % (RW * PER) * (16 / PER), n = tile * RW * 16 + c;
      if (n >= N) continue;
      const float v = total(m, c);
      if (EPI == LR_GLU) {
        reinterpret_cast<bf16*>(y)[(size_t)m * ldy + n / 2] = __float2bfloat16(glu_x(v, total(m, c + 1), ex.act, ex.limit));
      } else if (EPI == LR_SIDE) {
        const int id = ex.ids[m];
        float o = 0.f;
        if (n < ex.dim && id >= 0 && id < ex.vocab) o = gelu_tanh_x(v) * __bfloat162float(ex.side[(size_t)id * ex.ld_side + ex.off + n]);
        reinterpret_cast<bf16*>(y)[(size_t)m * ldy + n] = __float2bfloat16(o);
      } else if (EPI == LR_STORE && n >= ex.n_split) {
        ex.y2[(size_t)m * ex.ldy2 + n - ex.n_split] = v;
      } else if (EPI == LR_STORE) reinterpret_cast<bf16*>(y)[(size_t)m * ldy + n] = __float2bfloat16(n < ex.n_act ? act_x(v, ex.act) : v);
      else if (EPI == LR_STORE_F32) reinterpret_cast<float*>(y)[(size_t)m * ldy + n] = ex.cap > 0.f ? ex.cap * tanhf(v / ex.cap) : v;
      else reinterpret_cast<float*>(y)[(size_t)m * ldy + n] += v;
    }
    __syncthreads();
  }
  asm volatile("cp.async.wait_all;" ::: "memory");
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

// Most rows the projection takes for K columns (0: none): the staged rows and a two-stage ring fit shared memory.
TRL_API int trl_linear_rows_max(int K) {
  return max(0, min(16, (LR_SMEM - LR_WARPS * 2 * LR_SLOT) / ((K + LR_PAD) * 2)));
}

// x: bf16 [M, ldx], or the fp32 stream when norm_w is given (its row norm counts n_norm columns).  w: bf16 [N, K],
// K a multiple of 64.  epi: 0 store bf16, 1 store fp32, 2 add to fp32.  M <= trl_linear_rows_max(K).
static int lr_launch(const void* x, int ldx, const void* w, const void* norm_w, float eps, int n_norm, void* y, int ldy,
                     int M, int N, int K, int epi, const LrExtra& ex, void* stream) {
  if (M < 1 || N < 1 || K < 64 || K % 64 || M > trl_linear_rows_max(K) || ldx % 8 || epi < 0 || epi > 4 ||
      (norm_w && n_norm < 1) || ((uintptr_t)x & 15) || ((uintptr_t)w & 15))
    return (int)cudaErrorInvalidValue;
  const int groups = (N + 15) / 16;
  // split K over the warps of a block: shares of at least 16 steps, more splits where there are few rows
  int KW = 1;
  while (KW < LR_WARPS && (K / 32 / (2 * KW) >= 16 || (long)groups * KW < 2L * lr_sms() * LR_WARPS)) KW *= 2;
  const int RW = LR_WARPS / KW, n_tiles = (groups + RW - 1) / RW, grid = min(n_tiles, lr_sms());
  const size_t xb = (size_t)M * (ex.x2 ? 2 : 1) * (K + LR_PAD) * sizeof(bf16);
  if (xb + (size_t)LR_WARPS * 2 * LR_SLOT > (size_t)LR_SMEM) return (int)cudaErrorInvalidValue;
  const int nt = M <= 8 ? 1 : 2, depth = xb + LR_WARPS * 4 * LR_SLOT <= LR_SMEM ? 4 : 2;
  const size_t smem = xb + (size_t)LR_WARPS * depth * LR_SLOT;
  cudaError_t e = cudaErrorInvalidValue;
#define LR_CASE(NO, NTT, EP, DE)                                                                                        \
  if ((norm_w != nullptr) == NO && nt == NTT && epi == EP && depth == DE) {                                             \
    auto kern = linear_rows_kernel<NO, NTT, EP, DE>;                                                                    \
    static bool configured = false;                                                                                     \
    if (!configured) {                                                                                                  \
      e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, LR_SMEM);                             \
      if (e != cudaSuccess) return (int)e;                                                                              \
      cudaFuncSetAttribute(kern, cudaFuncAttributePreferredSharedMemoryCarveout, 100);                                  \
      configured = true;                                                                                                \
    }                                                                                                                   \
    e = trl_launch(kern, dim3(grid), dim3(LR_THREADS), smem, (cudaStream_t)stream, x, ldx, (const bf16*)w,              \
                   (const float*)norm_w, eps, n_norm, y, ldy, M, N, K, KW, n_tiles, ex);                                    \
  }
#define LR_BOTH(NO, NTT, EP) LR_CASE(NO, NTT, EP, 2) LR_CASE(NO, NTT, EP, 4)
  LR_BOTH(true, 1, LR_STORE) LR_BOTH(true, 1, LR_STORE_F32) LR_BOTH(true, 2, LR_STORE) LR_BOTH(true, 2, LR_STORE_F32)
  LR_BOTH(false, 1, LR_STORE) LR_BOTH(false, 1, LR_STORE_F32) LR_BOTH(false, 1, LR_ADD_F32)
  LR_BOTH(false, 2, LR_STORE) LR_BOTH(false, 2, LR_STORE_F32) LR_BOTH(false, 2, LR_ADD_F32)
  LR_BOTH(false, 1, LR_GLU) LR_BOTH(false, 2, LR_GLU) LR_BOTH(false, 1, LR_SIDE) LR_BOTH(false, 2, LR_SIDE)
#undef LR_BOTH
#undef LR_CASE
  return (int)e;
}

TRL_API int trl_linear_rows(const void* x, int ldx, const void* w, const void* norm_w, float eps, int n_norm, void* y, int ldy,
                            int M, int N, int K, int epi, void* stream) {
  if (epi > 2) return (int)cudaErrorInvalidValue;
  LrExtra ex = {};
  ex.n_split = 1 << 30;
  return lr_launch(x, ldx, w, norm_w, eps, n_norm, y, ldy, M, N, K, epi, ex, stream);
}

// Rows n < n_split as bf16 into y, the others as fp32 into y2 (both row-major, their own leading dimensions).
TRL_API int trl_linear_rows_split(const void* x, int ldx, const void* w, void* y, int ldy, int n_split, void* y2, int ldy2, int M, int N,
                                  int K, void* stream) {
  if (!y2 || n_split < 0) return (int)cudaErrorInvalidValue;
  LrExtra ex = {};
  ex.y2 = (float*)y2, ex.ldy2 = ldy2, ex.n_split = n_split;
  return lr_launch(x, ldx, w, nullptr, 0.f, 0, y, ldy, M, N, K, LR_STORE, ex, stream);
}

// The same with act (ACT_* of packed.cuh) on rows n < n_act, and rows n >= n_x2 (a multiple of 16) reading x2 (ldx, too; null: all read
// x).  With x2, 2 M rows must fit trl_linear_rows_max(K).
TRL_API int trl_linear_rows_mix(const void* x, int ldx, const void* x2, int n_x2, const void* w, void* y, int ldy, int n_split, void* y2, int ldy2,
                                int M, int N, int K, int n_act, int act, void* stream) {
  if (n_split < 0 || (n_split < N && !y2) || (n_split > 0 && !y) || n_act < 0 || n_act > n_split || act < ACT_NONE || act > ACT_GELU_ERF ||
      (x2 && (n_x2 % 16 || n_x2 < 0 || ((uintptr_t)x2 & 15))))
    return (int)cudaErrorInvalidValue;
  LrExtra ex = {};
  ex.y2 = (float*)y2, ex.ldy2 = ldy2, ex.n_split = n_split, ex.n_act = n_act, ex.act = act, ex.x2 = (const bf16*)x2, ex.n_x2 = n_x2;
  return lr_launch(x, ldx, w, nullptr, 0.f, 0, y, ldy, M, N, K, LR_STORE, ex, stream);
}

// y[m, n] = cap tanh((x W^T) / cap) in fp32.
TRL_API int trl_linear_rows_cap(const void* x, int ldx, const void* w, void* y, int ldy, int M, int N, int K, float cap, void* stream) {
  if (!(cap > 0.f)) return (int)cudaErrorInvalidValue;
  LrExtra ex = {};
  ex.cap = cap;
  return lr_launch(x, ldx, w, nullptr, 0.f, 0, y, ldy, M, N, K, LR_STORE_F32, ex, stream);
}

// w: rows 2j = gate_j, 2j + 1 = up_j; y: bf16 [M, N / 2].  act: GLU_* of packed.cuh.
TRL_API int trl_linear_rows_glu(const void* x, int ldx, const void* w, void* y, int ldy, int M, int N, int K, int act, float limit,
                                void* stream) {
  if (N % 2 || act < GLU_CLAMPED || act > GLU_GELU) return (int)cudaErrorInvalidValue;
  LrExtra ex = {};
  ex.act = act, ex.limit = limit;
  return lr_launch(x, ldx, w, nullptr, 0.f, 0, y, ldy, M, N, K, LR_GLU, ex, stream);
}

// y[m, n] = gelu(x W^T) * side[ids[m], off + n] for n < dim, 0 past it.
TRL_API int trl_linear_rows_side(const void* x, int ldx, const void* w, void* y, int ldy, int M, int N, int K, const void* ids, const void* side,
                                 long ld_side, int off, int dim, int vocab, void* stream) {
  if (!ids || !side || dim > N || off < 0 || off + dim > ld_side) return (int)cudaErrorInvalidValue;
  LrExtra ex = {};
  ex.ids = (const int*)ids, ex.side = (const bf16*)side, ex.ld_side = ld_side, ex.off = off, ex.dim = dim, ex.vocab = vocab;
  return lr_launch(x, ldx, w, nullptr, 0.f, 0, y, ldy, M, N, K, LR_SIDE, ex, stream);
}
