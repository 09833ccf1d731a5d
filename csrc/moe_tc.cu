// Expert projections of many rows on tcgen05 (kind::f16, bf16 operands, fp32 accumulation in TMEM).
//
//   UP    out[r, j] = act(W[e, 2j] x[r]) * (W[e, 2j + 1] x[r])      bf16, rows ordered by expert (moe_plan_kernel)
//   DOWN  out[r, n] = W[e, n] x[r]                                  bf16
//   ACT   out[r, n] = act(W[e, n] x[r])                             bf16
//
// A tile is 128 weight rows (the MMA's A operand: TMEM lanes) by up to 256 rows of one expert (its B operand: TMEM columns).  The
// instruction's N follows the rows an expert really has, in steps of 16, so a short expert costs what its rows cost.  K goes by in
// blocks of 64 (128-byte rows, 128-byte swizzle) through a ring of four stages filled by TMA; two accumulators of 256 columns let the
// epilogue of a tile run under the products of the next.  Blocks are persistent; neighbours work on the same rows, so that an
// expert's rows and weights are read from L2 by those after the first.
//
// Warp roles (320 threads): warp 0 = TMA producer, warp 1 = TMEM owner and MMA issuer, warps 2..9 = epilogue (two per TMEM lane
// quadrant, 128 columns each).  Every mbarrier wait is bounded (error word, abort flag, TMEM freed).
// Reference parity: the reference has dense feed-forwards only (no counterpart).
#include <cuda.h>

#include "moe.cuh"
#include "tcgen05.cuh"

namespace {

constexpr int MT_M = 128, MT_N = 256, MT_KB = 128;            // weight rows, expert rows, bytes of K per stage
constexpr int MT_BOX = 64;                                    // rows of a copy of the B operand
constexpr int MT_STAGES = 4, MT_A_BYTES = MT_M * MT_KB, MT_STAGE_BYTES = MT_A_BYTES + MT_N * MT_KB;
constexpr int MT_THREADS = 320, MT_EPI = MT_THREADS - 64;

struct TcArgs {
  const MoeItem* items;
  const int* n_items;
  bf16* out;
  int N, nkb, ldo, act, per_item;
};

__device__ __forceinline__ void tc_mma_bf16_lh(uint32_t d_tmem, uint32_t alo, uint32_t blo, uint32_t hi, uint32_t idesc, uint32_t accumulate) {
  asm volatile(
      "{ .reg .pred p; .reg .b64 da, db;\n"
      "  mov.b64 da, {%1, %3}; mov.b64 db, {%2, %3};\n"
      "  setp.ne.b32 p, %5, 0;\n"
      "  tcgen05.mma.cta_group::1.kind::f16 [%0], da, db, %4, p; }\n"
      ::"r"(d_tmem), "r"(alo), "r"(blo), "r"(hi), "r"(idesc), "r"(accumulate)
      : "memory");
}

template <int KIND>
__global__ void __launch_bounds__(MT_THREADS, 1)
moe_tc_kernel(const __grid_constant__ CUtensorMap map_w, const __grid_constant__ CUtensorMap map_x, const TcArgs p) {
  extern __shared__ unsigned char mt_smem[];
  unsigned char* smem = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(mt_smem) + 1023) & ~(uintptr_t)1023);
  uint64_t* bars = reinterpret_cast<uint64_t*>(smem + (size_t)MT_STAGES * MT_STAGE_BYTES);
  // bars: [0, S) full, [S, 2S) empty, 2S + {0, 1} accumulator full, 2S + {2, 3} accumulator empty
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 2 * MT_STAGES + 4);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const uint32_t bar0 = smem_u32(bars);
  auto full = [&](int s) { return bar0 + 8u * s; };
  auto empty = [&](int s) { return bar0 + 8u * (MT_STAGES + s); };
  auto acc_full = [&](int b) { return bar0 + 8u * (2 * MT_STAGES + b); };
  auto acc_empty = [&](int b) { return bar0 + 8u * (2 * MT_STAGES + 2 + b); };
  if (threadIdx.x == 0) {
    for (int s = 0; s < MT_STAGES; ++s) mbar_init(full(s), 1), mbar_init(empty(s), 1);
    for (int b = 0; b < 2; ++b) mbar_init(acc_full(b), 1), mbar_init(acc_empty(b), MT_EPI);
    *abort_flag = 0;
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "r"(2 * MT_N) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem_base = *tmem_slot;
  pdl_launch_dependents(66);
  pdl_wait();
  const int n_work = *p.n_items * p.per_item;

  if (warp == 0) {
    // ---------------- TMA producer ----------------
    if (lane == 0) {
      int st = 0;
      uint32_t ph = 0;
      long issued = 0;
      bool ok = true;
      for (int tile = blockIdx.x; ok && tile < n_work; tile += gridDim.x) {
        const MoeItem it = p.items[tile / p.per_item];
        const int w_row = it.expert * p.N + (tile % p.per_item) * MT_M, boxes = (it.n + MT_BOX - 1) / MT_BOX;
        for (int kb = 0; kb < p.nkb; ++kb, ++issued) {
          if (issued >= MT_STAGES && !(ok = mbar_wait(empty(st), ph ^ 1u, abort_flag))) break;
          const uint32_t dst = smem_u32(smem) + (uint32_t)st * MT_STAGE_BYTES;
          mbar_expect_tx(full(st), (uint32_t)(MT_A_BYTES + boxes * MT_BOX * MT_KB));
          tma_load_2d(dst, &map_w, kb * MT_KB, w_row, full(st));
          for (int b = 0; b < boxes; ++b)
            tma_load_2d(dst + MT_A_BYTES + b * MT_BOX * MT_KB, &map_x, kb * MT_KB, it.row0 + b * MT_BOX, full(st));
          if (++st == MT_STAGES) st = 0, ph ^= 1u;
        }
      }
    }
  } else if (warp == 1) {
    // ---------------- MMA issuer ----------------
    if (lane == 0) {
      const uint64_t d0 = desc_sw128(smem_u32(smem));
      const uint32_t lo0 = (uint32_t)d0, hi = (uint32_t)(d0 >> 32);
      int st = 0, count = 0;
      uint32_t ph = 0;
      bool ok = true;
      for (int tile = blockIdx.x; ok && tile < n_work; tile += gridDim.x, ++count) {
        const int buf = count & 1, n = (p.items[tile / p.per_item].n + 15) & ~15;
        // fp32 accumulator, bf16 x bf16, both K-major
        const uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(n >> 3) << 17) | ((uint32_t)(MT_M >> 4) << 24);
        if (count >= 2) {
          if (!(ok = mbar_wait(acc_empty(buf), (uint32_t)((count >> 1) - 1) & 1u, abort_flag))) break;
          tc_fence_after();
        }
        for (int kb = 0; kb < p.nkb; ++kb) {
          if (!(ok = mbar_wait(full(st), ph, abort_flag))) break;
          tc_fence_after();
          const uint32_t aoff = (uint32_t)st * (uint32_t)(MT_STAGE_BYTES >> 4), boff = aoff + (uint32_t)(MT_A_BYTES >> 4);
#pragma unroll
          for (int i = 0; i < 4; ++i)
            tc_mma_bf16_lh(tmem_base + (uint32_t)buf * MT_N, lo0 + aoff + i * 2, lo0 + boff + i * 2, hi, idesc, kb || i ? 1u : 0u);
          tc_commit(empty(st));
          if (++st == MT_STAGES) st = 0, ph ^= 1u;
        }
        if (ok) tc_commit(acc_full(buf));
      }
    }
  } else {
    // ---------------- epilogue (warps 2..9) ----------------
    const int quad = warp & 3, half = (warp - 2) >> 2;        // a warp may read only the TMEM lanes of its quadrant
    int count = 0;
    for (int tile = blockIdx.x; tile < n_work; tile += gridDim.x, ++count) {
      const int buf = count & 1;
      const MoeItem it = p.items[tile / p.per_item];
      const int f = (tile % p.per_item) * MT_M + quad * 32 + lane;               // weight row of this thread
      if (!__all_sync(0xffffffffu, mbar_wait(acc_full(buf), (uint32_t)(count >> 1) & 1u, abort_flag))) break;
      tc_fence_after();
      // lane pairs (2j, 2j + 1) trade values so that the even lane ends with both of column c, the odd one with both of column c + 1
      const bool odd = lane & 1;
      const int col = KIND == MOE_UP ? f >> 1 : f & ~1;
      bf16* out = p.out + (size_t)it.row0 * p.ldo + col;
      for (int c0 = half * (MT_N / 2); c0 < min(it.n, (half + 1) * (MT_N / 2)); c0 += 32) {
        uint32_t r[32];
        tc_ld32(tmem_base + ((uint32_t)(quad * 32) << 16) + (uint32_t)(buf * MT_N + c0), r);
        tc_wait_ld();
#pragma unroll
        for (int c = 0; c < 32; c += 2) {
          const float v0 = __uint_as_float(r[c]), v1 = __uint_as_float(r[c + 1]), mine = odd ? v1 : v0;
          const float other = __shfl_xor_sync(0xffffffffu, odd ? v0 : v1, 1);
          const float lo = odd ? other : mine, up = odd ? mine : other;          // weight rows f & ~1 and f | 1
          const int row = c0 + c + odd;
          if (row < it.n && f < p.N) {
            if (KIND == MOE_UP) out[(size_t)row * p.ldo] = __float2bfloat16(glu_x(lo, up, p.act, 0.f));
            else if (KIND == MOE_ACT) *reinterpret_cast<uint32_t*>(out + (size_t)row * p.ldo) = f2_to_bf162_bits(act_x(lo, p.act), act_x(up, p.act));
            else *reinterpret_cast<uint32_t*>(out + (size_t)row * p.ldo) = f2_to_bf162_bits(lo, up);
          }
        }
      }
      tc_fence_before();
      mbar_arrive(acc_empty(buf));
    }
  }

  // ---------------- teardown ----------------
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  if (*abort_flag) {
    const long long t0 = clock64();   // copies still in flight must land before the CTA's memory goes away
    while (clock64() - t0 < 2000000LL) {
    }
  }
  if (warp == 1)
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem_base), "r"(2 * MT_N) : "memory");
}

typedef CUresult (*EncodeTiledMt)(CUtensorMap*, CUtensorMapDataType, cuuint32_t, void*, const cuuint64_t*, const cuuint64_t*, const cuuint32_t*,
                                  const cuuint32_t*, CUtensorMapInterleave, CUtensorMapSwizzle, CUtensorMapL2promotion, CUtensorMapFloatOOBfill);
EncodeTiledMt g_encode_mt = nullptr;

// rows of row_bytes (a multiple of 128), boxes of box_rows x 128 bytes
int make_map(CUtensorMap* m, const void* base, uint64_t rows, uint64_t row_bytes, int box_rows) {
  if (!g_encode_mt) {
    void* fn = nullptr;
    cudaDriverEntryPointQueryResult q;
    if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &fn, cudaEnableDefault, &q) != cudaSuccess || !fn) return 1;
    g_encode_mt = (EncodeTiledMt)fn;
  }
  cuuint64_t dims[2] = {row_bytes, rows};
  cuuint64_t strides[1] = {row_bytes};
  cuuint32_t box[2] = {(cuuint32_t)MT_KB, (cuuint32_t)box_rows};
  cuuint32_t estr[2] = {1, 1};
  return g_encode_mt(m, CU_TENSOR_MAP_DATA_TYPE_UINT8, 2, const_cast<void*>(base), dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                     CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS ? 0 : 2;
}

}  // namespace

// Most rows of an item.
TRL_API int trl_moe_tc_tile() { return MT_N; }

// x: bf16 [rows, K] ordered by expert; w: bf16 [experts, N, K]; K a multiple of 64, N even.  kind 0: up (out [rows, N / 2]), 1: down,
// 2: plain up (out [rows, N]); ldo: a multiple of 2.  items: of at most trl_moe_tc_tile() rows each.
TRL_API int trl_moe_tc(const void* x, const void* w, void* out, int ldo, const void* items, const void* n_items, int rows, int experts, int N,
                       int K, int kind, int act, void* stream) {
  if (rows <= 0 || experts <= 0 || N <= 0 || N % 2 || K < 64 || K % 64 || ldo % 2 || kind < MOE_UP || kind > MOE_ACT || act < GLU_CLAMPED || act > (kind == MOE_ACT ? (int)ACT_GELU_ERF : (int)GLU_GELU) ||
      !items || !n_items || ((uintptr_t)x & 15) || ((uintptr_t)w & 15) || ((uintptr_t)out & 3))
    return (int)cudaErrorInvalidValue;
  CUtensorMap mw, mx;
  if (make_map(&mw, w, (uint64_t)experts * N, (uint64_t)K * 2, MT_M) || make_map(&mx, x, (uint64_t)rows, (uint64_t)K * 2, MT_BOX))
    return (int)cudaErrorInvalidValue;
  const size_t smem = (size_t)MT_STAGES * MT_STAGE_BYTES + 1024 + 256;
  static int sms = 0;
  if (!sms) {
    int dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    cudaError_t e = cudaFuncSetAttribute(moe_tc_kernel<MOE_UP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(moe_tc_kernel<MOE_ACT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(moe_tc_kernel<MOE_DOWN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
    if (e != cudaSuccess) {
      sms = 0;
      return (int)e;
    }
  }
  const TcArgs p = {(const MoeItem*)items, (const int*)n_items, (bf16*)out, N, K / 64, ldo, act, (N + MT_M - 1) / MT_M};
  if (kind == MOE_ACT) return (int)trl_launch(moe_tc_kernel<MOE_ACT>, dim3(sms), dim3(MT_THREADS), smem, (cudaStream_t)stream, mw, mx, p);
  if (kind == MOE_UP) return (int)trl_launch(moe_tc_kernel<MOE_UP>, dim3(sms), dim3(MT_THREADS), smem, (cudaStream_t)stream, mw, mx, p);
  return (int)trl_launch(moe_tc_kernel<MOE_DOWN>, dim3(sms), dim3(MT_THREADS), smem, (cudaStream_t)stream, mw, mx, p);
}
