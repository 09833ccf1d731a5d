// Causal softmax attention on the packed paged pool (page layout: tilerl_b200/kv.py, KvPage without factors), with the options of
// stream designs: a window, a soft cap on scores, a learned sink per head in the denominator, values of another width than keys.
//
//   qkv_prep_kernel             fused projection rows -> queries and cached keys / values of a token: an optional short convolution
//                               (earlier rows from the slot's ring), RMS norm with a weight over the whole projection or per head,
//                               rotation in halves or neighbouring pairs; or no norm, a bias, and values that turn like keys; two blocks
//                               per token.  Everything between the projection's
//                               rounding and the final one is fp32.
//   sm_attn_kernel<D, WM, WN>   tensor cores (mma.sync m16n8k16 bf16).  One block = (16 WM query rows, kv head, sequence, key split); a
//                               row is a (token, head of the group) pair.  Keys come 64 at a time (four pages) into a ring of stages,
//                               one bulk copy per page, from a producing warp; WN warps share a row tile and own 4 / WN pages of every
//                               stage each, with a running maximum of their own.  <.., 1, 4> serves decoding and short windows (up to
//                               16 rows), <.., 8, 1> and <256, 7, 1> prompts.  Pages outside a tile's window are not read.
//   sm_combine_kernel           merges the splits of a row.
//   sm_attn_plain_kernel        the same attention on CUDA cores: fp32 pools and heads beyond the tensor-core tiles.
//
// Scores, maxima, weights and sums are fp32; weights go into the value product as a bf16 pair (high part + rest).
// Reference parity: the reference's attention has no sink, cap, window or differing widths (no counterpart).
#include "packed.cuh"

namespace {

constexpr int TILE = 64, TPAGES = TILE / KVB;
constexpr long long SM_WAIT_CYCLES = 4000000000LL;
constexpr int SM_SMEM = 216 * 1024;
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float ex2_f(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
__device__ __forceinline__ float rcp_f(float x) {
  float y;
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}

// ---- queries, keys and values of a token -----------------------------------------------------------------
struct PrepArgs {
  const void* proj;                       // [T, ldp]; the layer's columns start at 0: [q | k | v]
  int ldp, heads, kv_heads, dim, dk, dv;  // true and padded widths
  int k0, v0, n_in, own;                  // first columns of keys and values, columns in all; own = 0: queries only
  int taps;                               // 0: no convolution
  const float* conv;                      // [taps, n_in]
  void* ring;                             // the layer's first column of slot 0
  long ring_slot;
  int ring_rows, ring_ld, write_ring;
  const float *q_norm, *k_norm;
  int norm_all;
  const double* freqs;
  int n_pairs, half;
  float eps;
  const int *positions, *seq_ids, *q_start, *slots, *slot_mapping;
  void* q;                                // [T, heads * dk]
  unsigned char* pages;
  int n_blocks;
  void* mid;                              // columns pad0 .. ldm - 1 are cleared
  int ldm, pad0;
  const float* bias;                      // [n_in], added behind the convolution; or null
  const double* vfreqs;                   // dv / 2 pairs (a value's halves) that turn with the position; or null
  float2* turn;                           // [T, dv / 2] their cos and sin
};

// grid (token, part): part 0 = queries, part 1 = keys and values.  Weights of a tick take the read-only path (they are constants).
template <typename T>
__global__ void __launch_bounds__(512) qkv_prep_kernel(const PrepArgs a) {
  constexpr int C = Chunk<T>::N;
  extern __shared__ __align__(16) float s_row[];           // the part's columns, then cos and sin, then a factor per head
  __shared__ float red[32];
  pdl_launch_dependents(50);
  const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nt = blockDim.x, nw = nt >> 5;
  const bool is_q = blockIdx.y == 0;
  const int base = is_q ? 0 : a.k0, cols = is_q ? a.k0 : a.n_in - a.k0, heads = is_q ? a.heads : a.kv_heads;
  float* s_cs = s_row + cols;
  float* s_fac = s_cs + 2 * a.n_pairs;
  float2* s_turn = reinterpret_cast<float2*>(s_fac + ((heads + 1) & ~1));
  pdl_wait();
  const int pos = a.positions[t], seq = a.seq_ids[t];
  const T* row = reinterpret_cast<const T*>(a.proj) + (size_t)t * a.ldp + base;
  T* ring = reinterpret_cast<T*>(a.ring) + (a.taps ? (size_t)a.slots[seq] * a.ring_slot + base : 0);
  const int t0 = a.q_start[seq];
  for (int i = tid; i < a.n_pairs; i += nt) pair_angle(pos, __ldg(a.freqs + i), 1.f, s_cs[2 * i], s_cs[2 * i + 1]);
  if (!is_q && a.vfreqs)
    for (int i = tid; i < a.dv / 2; i += nt) {
      float2 cs;
      pair_angle(pos, __ldg(a.vfreqs + i), 1.f, cs.x, cs.y);
      s_turn[i] = cs, a.turn[(size_t)t * (a.dv / 2) + i] = cs;
    }
  for (int c = tid * C; c < cols; c += nt * C) {
    const uint4 own = *reinterpret_cast<const uint4*>(row + c);
    float f[C];
    Chunk<T>::get(own, f);
    if (a.taps) {
      const float* w = a.conv + base + c;
      float acc[C];
#pragma unroll
      for (int e = 0; e < C; ++e) acc[e] = 0.f;
      for (int back = 0; back < a.taps && back <= pos; ++back) {
        if (back) {
          const T* src = t - back >= t0 ? row - (size_t)back * a.ldp + c : ring + (size_t)((pos - back) % a.ring_rows) * a.ring_ld + c;
          Chunk<T>::get(*reinterpret_cast<const uint4*>(src), f);
        }
#pragma unroll
        for (int e = 0; e < C; e += 4) {
          const float4 k = __ldg(reinterpret_cast<const float4*>(w + (size_t)(a.taps - 1 - back) * a.n_in + e));
          acc[e] = fmaf(f[e], k.x, acc[e]), acc[e + 1] = fmaf(f[e + 1], k.y, acc[e + 1]);
          acc[e + 2] = fmaf(f[e + 2], k.z, acc[e + 2]), acc[e + 3] = fmaf(f[e + 3], k.w, acc[e + 3]);
        }
      }
#pragma unroll
      for (int e = 0; e < C; ++e) f[e] = acc[e];
      if (a.write_ring) *reinterpret_cast<uint4*>(ring + (size_t)(pos % a.ring_rows) * a.ring_ld + c) = own;
    }
    if (a.bias) {
#pragma unroll
      for (int e = 0; e < C; e += 4) {
        const float4 b = __ldg(reinterpret_cast<const float4*>(a.bias + base + c + e));
        f[e] += b.x, f[e + 1] += b.y, f[e + 2] += b.z, f[e + 3] += b.w;
      }
    }
#pragma unroll
    for (int e = 0; e < C; e += 4) *reinterpret_cast<float4*>(s_row + c + e) = make_float4(f[e], f[e + 1], f[e + 2], f[e + 3]);
  }
  if (a.mid && is_q)
    for (int c = a.pad0 + tid; c < a.ldm; c += nt) reinterpret_cast<T*>(a.mid)[(size_t)t * a.ldm + c] = from_f<T>(0.f);
  __syncthreads();
  // ---- norm factors (padding columns hold zeros)
  if (!a.q_norm) {
    for (int h = tid; h < heads; h += nt) s_fac[h] = 1.f;
  } else if (a.norm_all) {
    float ss = 0.f;
    for (int c = tid * 4; c < heads * a.dk; c += nt * 4) {
      const float4 v = *reinterpret_cast<const float4*>(s_row + c);
      ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
    }
    ss = block_sum(ss, red);
    if (tid == 0) s_fac[0] = inv_rms(ss, heads * a.dim, a.eps);
  } else {
    for (int h = warp; h < heads; h += nw) {
      float ss = 0.f;
      for (int d = lane * 4; d < a.dk; d += 128) {
        const float4 v = *reinterpret_cast<const float4*>(s_row + h * a.dk + d);
        ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
      }
      ss = warp_sum(ss);
      if (lane == 0) s_fac[h] = inv_rms(ss, a.dim, a.eps);
    }
  }
  __syncthreads();
  // ---- turned rows, in chunks
  int slot = is_q ? 0 : a.slot_mapping[t];
  if (slot < 0) return;
  if (!is_q) slot = trl_checked(slot, a.n_blocks * KVB, 13);
  const int kch = a.dk / C, vch = a.dv / C, page_bytes = KVB * (kch + vch) * 16, r = slot & (KVB - 1);
  unsigned char* page0 = is_q ? nullptr : a.pages + (size_t)(slot / KVB) * a.kv_heads * page_bytes;
  const float* norm = is_q ? a.q_norm : a.k_norm;
  auto scaled = [&](const float* src, const float* w, float fac, int d, float (&o)[C]) {
#pragma unroll
    for (int e = 0; e < C; e += 4) {
      const float4 v = *reinterpret_cast<const float4*>(src + d + e);
      const float4 g = norm ? __ldg(reinterpret_cast<const float4*>(w + d + e)) : make_float4(1.f, 1.f, 1.f, 1.f);
      o[e] = v.x * fac * g.x, o[e + 1] = v.y * fac * g.y, o[e + 2] = v.z * fac * g.z, o[e + 3] = v.w * fac * g.w;
    }
  };
  for (int x = tid; x < heads * kch; x += nt) {
    const int h = x / kch, ci = x - h * kch, d0 = ci * C;
    const float* src = s_row + h * a.dk;
    const float* w = norm + (norm && a.norm_all ? h * a.dk : 0);
    const float fac = s_fac[norm && a.norm_all ? 0 : h];
    float o[C];
    scaled(src, w, fac, d0, o);
    if (d0 < 2 * a.n_pairs) {
      if (!a.half) {
#pragma unroll
        for (int e = 0; e < C; e += 2) {
          if (d0 + e < 2 * a.n_pairs) {
            const float2 cs = *reinterpret_cast<const float2*>(s_cs + d0 + e);
            const float u = o[e], v = o[e + 1];
            o[e] = fmaf(u, cs.x, -v * cs.y), o[e + 1] = fmaf(v, cs.x, u * cs.y);
          }
        }
      } else if (a.n_pairs % C == 0) {                      // a chunk turns with one other chunk
        const bool second = d0 >= a.n_pairs;
        const int p0 = second ? d0 - a.n_pairs : d0;
        float m[C];
        scaled(src, w, fac, second ? p0 : d0 + a.n_pairs, m);
#pragma unroll
        for (int e = 0; e < C; ++e) {
          const float2 cs = *reinterpret_cast<const float2*>(s_cs + 2 * (p0 + e));
          o[e] = second ? fmaf(o[e], cs.x, m[e] * cs.y) : fmaf(o[e], cs.x, -m[e] * cs.y);
        }
      } else {
#pragma unroll
        for (int e = 0; e < C; ++e) {
          const int d = d0 + e;
          if (d < 2 * a.n_pairs) {
            const bool second = d >= a.n_pairs;
            const int p = second ? d - a.n_pairs : d, m = second ? p : d + a.n_pairs;
            const float u = src[m] * fac * (norm ? w[m] : 1.f), c = s_cs[2 * p], s = s_cs[2 * p + 1];
            o[e] = second ? fmaf(o[e], c, u * s) : fmaf(o[e], c, -u * s);
          }
        }
      }
    }
    const uint4 out = Chunk<T>::put(o);
    if (is_q) {
      *reinterpret_cast<uint4*>(reinterpret_cast<T*>(a.q) + (size_t)t * a.k0 + h * a.dk + d0) = out;
    } else {
      uint4* kd = reinterpret_cast<uint4*>(page0 + (size_t)h * page_bytes);
      kd[r * kch + page_chunk(ci, r, kch)] = out;
    }
  }
  if (is_q) return;
  for (int x = tid; x < a.kv_heads * vch; x += nt) {
    const int h = x / vch, c = x - h * vch;
    const float* src = s_row + a.v0 - a.k0 + h * a.dv + c * C;
    float o[C];
#pragma unroll
    for (int e = 0; e < C; e += 4) {
      const float4 v = *reinterpret_cast<const float4*>(src + e);
      o[e] = v.x, o[e + 1] = v.y, o[e + 2] = v.z, o[e + 3] = v.w;
    }
    if (a.vfreqs) {                                         // a chunk turns with the one half a head away
      const int half = a.dv / 2, d0 = c * C;
      const bool second = d0 >= half;
      const float* other = second ? src - half : src + half;
      const float2* cs = s_turn + (second ? d0 - half : d0);
#pragma unroll
      for (int e = 0; e < C; ++e) o[e] = second ? fmaf(o[e], cs[e].x, other[e] * cs[e].y) : fmaf(o[e], cs[e].x, -other[e] * cs[e].y);
    }
    uint4* vd = reinterpret_cast<uint4*>(page0 + (size_t)h * page_bytes + KVB * kch * 16);
    vd[r * vch + page_chunk(c, r, vch)] = Chunk<T>::put(o);
  }
}

// ---- attention ------------------------------------------------------------------------------------------
struct SmArgs {
  const void* q;                       // [T, n_q * dk]
  const unsigned char* pages;          // [n_blocks, n_kv, page_bytes]
  int page_bytes, kch, vch, n_blocks;  // 16-byte chunks of a K / V row
  const int* table;
  int max_blocks;
  const int *q_start, *q_len, *positions;
  const float* sink;                   // per head, or null
  void* out;
  int ldo;
  float* part;                         // [T, n_q, n_splits, dv], relative to the maximum beside it
  float2* ml;                          // [T, n_q, n_splits] (maximum in powers of two, sum)
  int n_q, n_kv, n_splits, n_stages, window, min_len, max_len;
  float scale, cap, factor;
  const float2* turn;                  // [T, dv / 2]: finished rows are turned back by these (their halves pair up); or null
};

// Keys [lo, hi) that the rows [row0, row0 + rows) of a sequence see; lo is a page's first.
__device__ __forceinline__ int2 tile_keys(const SmArgs& a, int row0, int rows, int n_rows, int G, int q0) {
  const int hi = a.positions[q0 + (min(row0 + rows, n_rows) - 1) / G] + 1;
  const int lo = a.window > 0 ? max(0, a.positions[q0 + row0 / G] - a.window + 1) & ~(KVB - 1) : 0;
  return make_int2(lo, hi);
}
// A pair of a finished row, turned back by its query's angle.
__device__ __forceinline__ float2 turn_back(float u, float v, const float2& cs) {
  return make_float2(fmaf(u, cs.x, v * cs.y), fmaf(v, cs.x, -u * cs.y));
}
// Pages per split (a multiple of a stage), and splits that hold keys.
__device__ __forceinline__ int split_pages(int keys, int n_splits) {
  const int pages = (keys + KVB - 1) / KVB;
  const int want = max(1, min(n_splits, (keys + 2 * TILE - 1) / (2 * TILE)));
  return ((pages + want - 1) / want + TPAGES - 1) / TPAGES * TPAGES;
}
__device__ __forceinline__ int splits_used(int keys, int n_splits) {
  const int pages = (keys + KVB - 1) / KVB, pps = split_pages(keys, n_splits);
  return (pages + pps - 1) / pps;
}
// weight of a partial result with maximum m under the maximum `top` (both in powers of two)
__device__ __forceinline__ float rel_weight(float m, float top) { return m == -INFINITY ? 0.f : ex2_f(m - top); }
// (scale of sums taken under the maximum m, denominator) once the head's sink has joined
__device__ __forceinline__ float2 with_sink(float m, float l, const float* sink, int h) {
  if (!sink) return make_float2(1.f, l);
  const float s = sink[h] * LOG2E, top = fmaxf(m, s), e = rel_weight(m, top);
  return make_float2(e, fmaf(l, e, ex2_f(s - top)));
}

__device__ __forceinline__ uint32_t sm_try_wait(uint32_t bar, uint32_t parity) {
  uint32_t ok;
  asm volatile("{ .reg .pred p;\n"
               "  mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n"
               "  selp.u32 %0, 1, 0, p; }\n"
               : "=r"(ok) : "r"(bar), "r"(parity) : "memory");
  return ok;
}

// FULL: K and V rows are D wide, so every chunk place is a constant away from one of four addresses a thread keeps.
template <int D, int WM, int WN, bool FULL>
__global__ void __launch_bounds__((WM * WN + 1) * 32)
sm_attn_kernel(const SmArgs a) {
  constexpr int ROWS = 16 * WM, NP = TPAGES / WN, NWC = WM * WN, THREADS = (NWC + 1) * 32;
  extern __shared__ unsigned char sm_smem_raw[];
  __shared__ __align__(8) uint64_t s_bar[8];               // full[4], empty[4]
  __shared__ float s_m[WN][ROWS], s_l[WN][ROWS];
  __shared__ volatile int s_ok;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int kch = FULL ? D / 8 : a.kch, vch = FULL ? D / 8 : a.vch, page_bytes = FULL ? KVB * D * 4 : a.page_bytes;
  const uint32_t raw_a = (uint32_t)__cvta_generic_to_shared(sm_smem_raw);
  unsigned char* smem = sm_smem_raw + (((raw_a + 127u) & ~127u) - raw_a);
  const uint32_t bar_a = (uint32_t)__cvta_generic_to_shared(s_bar);
  if (threadIdx.x == 0) {
    for (int st = 0; st < a.n_stages; ++st) {
      asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(bar_a + 8u * st));
      asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar_a + 32u + 8u * st), "r"(NWC));
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    s_ok = 1;
  }
  pdl_enter(51);
  pdl_wait();
  const int n_tiles_x = gridDim.x / a.n_splits;
  const int tile = n_tiles_x - 1 - (int)blockIdx.x / a.n_splits, split = blockIdx.x % a.n_splits;   // longest key ranges first
  const int kvh = blockIdx.y, seq = blockIdx.z;
  const int G = a.n_q / a.n_kv, T = a.q_len[seq], n_rows = T * G, row0 = tile * ROWS;
  if (T < a.min_len || T > a.max_len || row0 >= n_rows) return;
  const int q0 = a.q_start[seq];
  const int2 range = tile_keys(a, row0, ROWS, n_rows, G, q0);
  const int pps = split_pages(range.y - range.x, a.n_splits), used = splits_used(range.y - range.x, a.n_splits);
  if (split >= used) return;
  const int lo = range.x + split * pps * KVB, hi = min(range.y, range.x + (split + 1) * pps * KVB);
  const int n_tiles = (hi - lo + TILE - 1) / TILE;
  const int qld = kch * 16 + 16;                          // Q row stride in bytes: an odd number of 16-byte units
  const uint32_t q_a = (uint32_t)__cvta_generic_to_shared(smem);
  const int q_bytes = (ROWS * qld + 127) / 128 * 128, stage_bytes = TPAGES * page_bytes;
  unsigned char* ring = smem + q_bytes;
  const uint32_t ring_a = q_a + q_bytes;
  const int v_off = KVB * kch * 16;

  for (int x = threadIdx.x; x < ROWS * kch; x += THREADS) {
    const int r = x / kch, c = x % kch, row = row0 + r;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (row < n_rows)
      v = *reinterpret_cast<const uint4*>(reinterpret_cast<const bf16*>(a.q) + ((size_t)(q0 + row / G) * a.n_q + kvh * G + row % G) * (kch * 8) + c * 8);
    *reinterpret_cast<uint4*>(smem + r * qld + c * 16) = v;
  }
  {
    // The last page brings only the V rows that exist (the pool may hold anything past them, and 0 x V must be
    // 0): if nothing was copied into that place before, its tail starts as zeros.
    const int last = n_tiles - 1, tail = hi & (KVB - 1);
    if (tail && last < a.n_stages) {
      const int pg = ((hi - 1 - lo) / KVB) % TPAGES;
      unsigned char* v = ring + last * stage_bytes + pg * page_bytes + v_off;
      for (int x = tail * vch + threadIdx.x; x < KVB * vch; x += THREADS)
        *reinterpret_cast<uint4*>(v + x * 16) = make_uint4(0u, 0u, 0u, 0u);
    }
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  __syncthreads();

  auto bounded_wait = [&](uint32_t bar, uint32_t parity, int what) {
    if (sm_try_wait(bar, parity)) return true;
    const long long t_begin = clock64();
    for (uint32_t it = 1; !sm_try_wait(bar, parity); ++it) {
      if ((it & 63) == 0) {
        if (!s_ok) return false;
        if (clock64() - t_begin > SM_WAIT_CYCLES) {
          trl_set_error(TRL_ERR_MBAR_TIMEOUT, (int)blockIdx.x, what, (int)parity);
          s_ok = 0;
          return false;
        }
      }
    }
    return true;
  };

  const int wm = warp / WN, wn = warp % WN;
  float o[D / 8][4];
#pragma unroll
  for (int i = 0; i < D / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  float mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.f, 0.f};

  if (warp == NWC) {
    // ---------------- producer ----------------
    const int* table = a.table + (size_t)seq * a.max_blocks;
    int st = 0;
    uint32_t ph = 0;
    for (int kt = 0; kt < n_tiles; ++kt) {
      if (kt >= a.n_stages && !bounded_wait(bar_a + 32u + 8u * st, ph ^ 1u, 610 + st)) break;
      const int j0 = lo + kt * TILE, n_pg = min(TPAGES, (hi - j0 + KVB - 1) / KVB);
      uint32_t bytes = 0;
      const unsigned char* src = nullptr;
      if (lane < n_pg) {
        const int p = j0 / KVB + lane, keys = min(KVB, hi - p * KVB);
        const int blk = trl_checked(table[p], a.n_blocks, 14);
        src = a.pages + ((size_t)blk * a.n_kv + kvh) * page_bytes;
        bytes = (uint32_t)(v_off + keys * vch * 16);
      }
      const uint32_t total = __reduce_add_sync(0xffffffffu, bytes);
      const uint32_t full = bar_a + 8u * st;
      if (lane == 0) asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(full), "r"(total) : "memory");
      __syncwarp();
      if (lane < n_pg)
        asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                     ::"r"(ring_a + st * stage_bytes + lane * page_bytes), "l"(src), "r"(bytes), "r"(full) : "memory");
      if (++st == a.n_stages) st = 0, ph ^= 1u;
    }
  } else {
    // ---------------- consumers ----------------
    const int r_lo = wm * 16 + (lane >> 2);                 // fragment rows r_lo and r_lo + 8 of the block
    const int win = a.window > 0 ? a.window : 1 << 30;
    int pos[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int row = row0 + r_lo + 8 * i;
      pos[i] = row < n_rows ? a.positions[q0 + row / G] : -1;
    }
    const int my_rows = min(16, n_rows - row0 - wm * 16);   // the warp's rows: positions p_first .. p_last
    const int p_first = my_rows > 0 ? a.positions[q0 + (row0 + wm * 16) / G] : 0;
    const int p_last = my_rows > 0 ? a.positions[q0 + (row0 + wm * 16 + my_rows - 1) / G] : 0;
    const int my_hi = my_rows > 0 ? min(hi, p_last + 1) : 0, my_lo = p_first - win + 1;      // keys outside [my_lo, my_hi) are not seen
    const float s_in = a.cap > 0.f ? a.scale / a.cap * (2.f * LOG2E) : a.scale * LOG2E, s_cap = a.cap * LOG2E;
    const uint32_t qa = q_a + (wm * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * qld + (lane >> 4) * 16;
    const int kr = (lane & 7) + (lane >> 4) * 8, kcl = (lane >> 3) & 1;
    const int vr = (lane & 7) + ((lane >> 3) & 1) * 8, vcl = lane >> 4;
    uint32_t ka[4], va[4];                                  // FULL: offsets of chunks kcl + {0, 2, 4, 6} of this lane's rows
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      ka[i] = (uint32_t)(kr * kch * 16 + ((kcl ^ (kr & 7) ^ (2 * i)) << 4));
      va[i] = (uint32_t)(v_off + vr * vch * 16 + ((vcl ^ (vr & 7) ^ (2 * i)) << 4));
    }
    const int krot = kr % kch, vrot = vr % vch;
    auto place = [](int c, int r, int rot, int n) {         // page_chunk without a division (rot = r % n)
      const int x = c + rot;
      return n % 8 == 0 ? c ^ (r & 7) : (x >= n ? x - n : x);
    };
    auto k_off = [&](int c) {                               // c even
      if constexpr (FULL) return ka[(c >> 1) & 3] + (uint32_t)((c >> 3) * 128);
      else return (uint32_t)((kr * kch + place(c + kcl, kr, krot, kch)) * 16);
    };
    auto v_at = [&](int c) {
      if constexpr (FULL) return va[(c >> 1) & 3] + (uint32_t)((c >> 3) * 128);
      else return (uint32_t)(v_off + (vr * vch + place(c + vcl, vr, vrot, vch)) * 16);
    };
    int st = 0;
    uint32_t ph = 0;
    for (int kt = 0; kt < n_tiles; ++kt) {
      if (!bounded_wait(bar_a + 8u * st, ph, 600 + st)) break;
      const int jw = lo + kt * TILE + wn * NP * KVB;        // first key of this warp's pages
      if (jw < my_hi && jw + NP * KVB > my_lo) {
        const uint32_t base = ring_a + st * stage_bytes + wn * NP * page_bytes;
        // ---- scores of NP x 16 keys (pages past the range hold stale bytes: masked below)
        float sc[NP][2][4];
#pragma unroll
        for (int p = 0; p < NP; ++p)
#pragma unroll
          for (int n8 = 0; n8 < 2; ++n8) sc[p][n8][0] = sc[p][n8][1] = sc[p][n8][2] = sc[p][n8][3] = 0.f;
#pragma unroll
        for (int kk = 0; kk < D / 16; ++kk) {
          if (FULL || kk * 2 < kch) {
            uint32_t qv[4];
            ldsm4(qv, qa + kk * 32);
            const uint32_t ko = k_off(kk * 2);
#pragma unroll
            for (int p = 0; p < NP; ++p) {
              uint32_t b[4];
              ldsm4(b, base + p * page_bytes + ko);
              mma16(sc[p][0], qv, b[0], b[1]);
              mma16(sc[p][1], qv, b[2], b[3]);
            }
          }
        }
        // ---- scores in powers of two, running maximum
        float top[2] = {mx[0], mx[1]};
#pragma unroll
        for (int p = 0; p < NP; ++p) {
          const int j0 = jw + p * KVB;
          const bool edge = j0 + KVB - 1 > p_first || j0 <= p_last - win;      // some row does not see all of this page
#pragma unroll
          for (int n8 = 0; n8 < 2; ++n8)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
              float s = sc[p][n8][e] * s_in;
              if (a.cap > 0.f) s = fmaf(-2.f * s_cap, rcp_f(1.f + ex2_f(s)), s_cap);          // cap tanh(x / cap)
              if (edge) {                                   // (a select: stale bytes past the range may be anything)
                const int j = j0 + n8 * 8 + (lane & 3) * 2 + (e & 1), back = pos[e >> 1] - j;
                s = back >= 0 && back < win ? s : -INFINITY;
              }
              sc[p][n8][e] = s;
              top[e >> 1] = fmaxf(top[e >> 1], s);
            }
        }
        float ref[2];
        bool moved = false;
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          top[i] = fmaxf(top[i], __shfl_xor_sync(0xffffffffu, top[i], 1));
          top[i] = fmaxf(top[i], __shfl_xor_sync(0xffffffffu, top[i], 2));
          ref[i] = top[i] == -INFINITY ? 0.f : top[i];
          moved |= top[i] > mx[i];
        }
        if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const float f = rel_weight(mx[i], ref[i]);
            sum[i] *= f, mx[i] = top[i];
#pragma unroll
            for (int nd = 0; nd < D / 8; ++nd) o[nd][2 * i] *= f, o[nd][2 * i + 1] *= f;
          }
        }
        // ---- weights, and O += W V
#pragma unroll
        for (int p = 0; p < NP; ++p) {
          const int j0 = jw + p * KVB;
          if (j0 < my_hi && j0 + KVB > my_lo) {
            uint32_t wh[4], wl[4];
#pragma unroll
            for (int n8 = 0; n8 < 2; ++n8)
#pragma unroll
              for (int i = 0; i < 2; ++i) {
                const float w0 = ex2_f(sc[p][n8][2 * i] - ref[i]), w1 = ex2_f(sc[p][n8][2 * i + 1] - ref[i]);
                sum[i] += w0 + w1;
                split2(w0, w1, wh[n8 * 2 + i], wl[n8 * 2 + i]);
              }
            const uint32_t vb = base + p * page_bytes;
#pragma unroll
            for (int nd = 0; nd < D / 8; nd += 2) {
              if (FULL || nd < vch) {
                uint32_t b[4];
                ldsm4t(b, vb + v_at(nd));
                mma16(o[nd], wh, b[0], b[1]);
                mma16(o[nd + 1], wh, b[2], b[3]);
                mma16(o[nd], wl, b[0], b[1]);
                mma16(o[nd + 1], wl, b[2], b[3]);
              }
            }
          }
        }
      }
      __syncwarp();
      if (lane == 0) asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar_a + 32u + 8u * st) : "memory");
      if (++st == a.n_stages) st = 0, ph ^= 1u;
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 1);
      sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 2);
    }
  }
  __syncthreads();
  pdl_trigger();                                            // (not earlier: waiting blocks would take the room of working ones)
  if (!s_ok) {                                              // copies may still be in flight towards this block
    const long long t_begin = clock64();
    while (clock64() - t_begin < 2000000LL) {
    }
  }
  const int dv = vch * 8;
  auto cell = [&](int row) { return (size_t)(q0 + row / G) * a.n_q + kvh * G + row % G; };
  auto dst_part = [&](int row) { return a.part + (cell(row) * a.n_splits + split) * dv; };
  auto dst_out = [&](int row) { return reinterpret_cast<bf16*>(a.out) + (size_t)(q0 + row / G) * a.ldo + (size_t)(kvh * G + row % G) * dv; };
  if constexpr (WN == 1) {
    if (warp == NWC) return;
    if (a.turn && used == 1) {                              // a pair's halves meet in the (idle) ring
      const int lds = dv + 8, half = dv / 2;
      float* so = reinterpret_cast<float*>(ring) + (size_t)wm * 16 * lds;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int r = (lane >> 2) + 8 * i, row = row0 + wm * 16 + r;
        if (row >= n_rows) continue;
        const float2 f = with_sink(mx[i], sum[i], a.sink, kvh * G + row % G);
        const float g = f.x / f.y * a.factor;
#pragma unroll
        for (int nd = 0; nd < D / 8; ++nd)
          if (FULL || nd < vch) *reinterpret_cast<float2*>(so + r * lds + nd * 8 + (lane & 3) * 2) = make_float2(o[nd][2 * i] * g, o[nd][2 * i + 1] * g);
      }
      __syncwarp();
      for (int x = lane; x < 16 * (half / 2); x += 32) {
        const int r = x / (half / 2), m = x % (half / 2) * 2, row = row0 + wm * 16 + r;
        if (row >= n_rows) break;
        const float4 cs = *reinterpret_cast<const float4*>(a.turn + (size_t)(q0 + row / G) * half + m);
        const float2 u = *reinterpret_cast<const float2*>(so + r * lds + m), v = *reinterpret_cast<const float2*>(so + r * lds + half + m);
        const float2 p0 = turn_back(u.x, v.x, make_float2(cs.x, cs.y)), p1 = turn_back(u.y, v.y, make_float2(cs.z, cs.w));
        *reinterpret_cast<uint32_t*>(dst_out(row) + m) = f2_to_bf162_bits(p0.x, p1.x);
        *reinterpret_cast<uint32_t*>(dst_out(row) + half + m) = f2_to_bf162_bits(p0.y, p1.y);
      }
      return;
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int row = row0 + wm * 16 + (lane >> 2) + 8 * i;
      if (row >= n_rows) continue;
      const float2 f = with_sink(mx[i], sum[i], a.sink, kvh * G + row % G);
      const float g = used == 1 ? f.x / f.y * a.factor : 1.f;
      if (used > 1 && (lane & 3) == 0) a.ml[cell(row) * a.n_splits + split] = make_float2(mx[i], sum[i]);
#pragma unroll
      for (int nd = 0; nd < D / 8; ++nd) {
        if (FULL || nd < vch) {
          const int d = nd * 8 + (lane & 3) * 2;
          if (used == 1) *reinterpret_cast<uint32_t*>(dst_out(row) + d) = f2_to_bf162_bits(o[nd][2 * i] * g, o[nd][2 * i + 1] * g);
          else *reinterpret_cast<float2*>(dst_part(row) + d) = make_float2(o[nd][2 * i], o[nd][2 * i + 1]);
        }
      }
    }
  } else {
    // the WN warps of a row tile saw different keys: merge them in order, through the (idle) ring
    float* so = reinterpret_cast<float*>(ring);             // [WN][ROWS][dv]
    if (warp < NWC) {
      const int r = wm * 16 + (lane >> 2);
      if ((lane & 3) == 0) s_m[wn][r] = mx[0], s_m[wn][r + 8] = mx[1], s_l[wn][r] = sum[0], s_l[wn][r + 8] = sum[1];
#pragma unroll
      for (int nd = 0; nd < D / 8; ++nd) {
        if (FULL || nd < vch) {
          const int d = nd * 8 + (lane & 3) * 2;
          *reinterpret_cast<float2*>(so + ((size_t)wn * ROWS + r) * dv + d) = make_float2(o[nd][0], o[nd][1]);
          *reinterpret_cast<float2*>(so + ((size_t)wn * ROWS + r + 8) * dv + d) = make_float2(o[nd][2], o[nd][3]);
        }
      }
    }
    __syncthreads();
    const int rows = min(ROWS, n_rows - row0), half = dv / 2;
    const bool turned = a.turn && used == 1;                // a thread takes both of a pair
    const int cols = turned ? half : dv;
    for (int x = threadIdx.x; x < rows * cols; x += THREADS) {
      const int r = x / cols, d = x % cols, row = row0 + r;
      float top = -INFINITY, l = 0.f, v = 0.f, v2 = 0.f;
#pragma unroll
      for (int k = 0; k < WN; ++k) top = fmaxf(top, s_m[k][r]);
#pragma unroll
      for (int k = 0; k < WN; ++k) {
        const float e = rel_weight(s_m[k][r], top);
        l = fmaf(s_l[k][r], e, l);
        v = fmaf(so[((size_t)k * ROWS + r) * dv + d], e, v);
        if (turned) v2 = fmaf(so[((size_t)k * ROWS + r) * dv + half + d], e, v2);
      }
      if (turned) {
        const float2 f = with_sink(top, l, a.sink, kvh * G + row % G);
        const float g = f.x / f.y * a.factor;
        const float2 p = turn_back(v * g, v2 * g, a.turn[(size_t)(q0 + row / G) * half + d]);
        dst_out(row)[d] = __float2bfloat16(p.x), dst_out(row)[half + d] = __float2bfloat16(p.y);
      } else if (used == 1) {
        const float2 f = with_sink(top, l, a.sink, kvh * G + row % G);
        dst_out(row)[d] = __float2bfloat16(v * (f.x / f.y * a.factor));
      } else {
        dst_part(row)[d] = v;
        if (d == 0) a.ml[cell(row) * a.n_splits + split] = make_float2(top, l);
      }
    }
  }
}

// grid (token, head): merges the partial rows of a launch whose row tiles were `rows` tall
constexpr int CB_THREADS = 256;
__global__ void __launch_bounds__(CB_THREADS) sm_combine_kernel(const SmArgs a, const int* seq_ids, int rows) {
  __shared__ float s_w[64];                                 // weight of each split
  __shared__ float2 s_v[CB_THREADS];
  pdl_launch_dependents(52);
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y, seq = seq_ids[t], T = a.q_len[seq];
  const int G = a.n_q / a.n_kv, q0 = a.q_start[seq];
  if (T < a.min_len || T > a.max_len || t - q0 >= T) return;
  const int row0 = ((t - q0) * G + h % G) / rows * rows;
  const int2 range = tile_keys(a, row0, rows, T * G, G, q0);
  const int used = splits_used(range.y - range.x, a.n_splits);
  if (used == 1) return;
  const int dv = a.vch * 8;
  const size_t cell = (size_t)t * a.n_q + h;
  const float2* ml = a.ml + cell * a.n_splits;
  const float* p = a.part + cell * a.n_splits * dv;
  // every warp on its own: all splits' maxima and sums (at most 64), two a lane
  const int lane = threadIdx.x & 31;
  const float2 none = make_float2(-INFINITY, 0.f), m0 = lane < used ? ml[lane] : none, m1 = lane + 32 < used ? ml[lane + 32] : none;
  const float top = warp_max(fmaxf(m0.x, m1.x)), w0 = rel_weight(m0.x, top), w1 = rel_weight(m1.x, top);
  const float2 f = with_sink(top, warp_sum(fmaf(m0.y, w0, m1.y * w1)), a.sink, h);
  const float g = f.x / f.y * a.factor;
  if (threadIdx.x < 32) s_w[lane] = w0, s_w[lane + 32] = w1;
  __syncthreads();
  // a thread: two columns of every n_g-th split; then the n_g sums of a column in order
  const int pairs = dv / 2, n_g = CB_THREADS / pairs, grp = threadIdx.x / pairs, d = threadIdx.x % pairs * 2;
  float2 v = make_float2(0.f, 0.f);
  if (grp < n_g) {
#pragma unroll 4
    for (int s = grp; s < used; s += n_g) {
      const float2 x = *reinterpret_cast<const float2*>(p + (size_t)s * dv + d);
      v.x = fmaf(x.x, s_w[s], v.x), v.y = fmaf(x.y, s_w[s], v.y);
    }
  }
  s_v[threadIdx.x] = v;
  __syncthreads();
  if (grp == 0)
    for (int k = 1; k < n_g; ++k) v.x += s_v[k * pairs + threadIdx.x].x, v.y += s_v[k * pairs + threadIdx.x].y;
  if (a.turn) {                                             // (uniform) a pair's halves meet in shared memory
    __syncthreads();
    s_v[threadIdx.x] = v;
    __syncthreads();
    if (grp == 0) {
      const bool second = d >= dv / 2;
      const float2 o = s_v[second ? threadIdx.x - pairs / 2 : threadIdx.x + pairs / 2];
      const float4 cs = *reinterpret_cast<const float4*>(a.turn + (size_t)t * (dv / 2) + (second ? d - dv / 2 : d));
      v = second ? make_float2(fmaf(v.x, cs.x, -o.x * cs.y), fmaf(v.y, cs.z, -o.y * cs.w)) : make_float2(fmaf(v.x, cs.x, o.x * cs.y), fmaf(v.y, cs.z, o.y * cs.w));
    }
  }
  if (grp) return;
  *reinterpret_cast<uint32_t*>(reinterpret_cast<bf16*>(a.out) + (size_t)t * a.ldo + (size_t)h * dv + d) = f2_to_bf162_bits(v.x * g, v.y * g);
}

// CUDA cores: one block = (16 query rows, kv head, sequence), a page of keys at a time; thread (r, c) forms the score of
// row r and key c and owns the output columns c, c + 16, ... of row r.
constexpr int F_ROWS = 16, F_MAXD = 512;
template <typename T>
__global__ void __launch_bounds__(256) sm_attn_plain_kernel(const SmArgs a) {
  constexpr int C = Chunk<T>::N;
  extern __shared__ float sf[];
  __shared__ float s_w[F_ROWS][KVB + 1];
  pdl_launch_dependents(53);
  pdl_wait();
  const int kvh = blockIdx.y, seq = blockIdx.z, G = a.n_q / a.n_kv, len = a.q_len[seq], n_rows = len * G, row0 = blockIdx.x * F_ROWS;
  if (row0 >= n_rows) return;
  const int q0 = a.q_start[seq], kch = a.kch, vch = a.vch, dk = kch * C, dv = vch * C;
  float* sq = sf;                                  // [16][dk + 1]
  float* sk = sq + F_ROWS * (dk + 1);              // [16][dk + 1]
  float* sv = sk + KVB * (dk + 1);                 // [16][dv]
  const int r = threadIdx.x >> 4, c = threadIdx.x & 15, row = row0 + r;
  const bool in = row < n_rows;
  const int t = in ? q0 + row / G : q0, h = kvh * G + (in ? row % G : 0);
  for (int d = c; d < dk; d += 16) sq[r * (dk + 1) + d] = in ? to_f(reinterpret_cast<const T*>(a.q)[((size_t)t * a.n_q + h) * dk + d]) : 0.f;
  const int pos = in ? a.positions[t] : -1, win = a.window > 0 ? a.window : 1 << 30;
  float acc[F_MAXD / 16], m = -INFINITY, l = 0.f;
#pragma unroll
  for (int i = 0; i < F_MAXD / 16; ++i) acc[i] = 0.f;
  const int2 range = tile_keys(a, row0, F_ROWS, n_rows, G, q0);
  for (int p = range.x / KVB; p * KVB < range.y; ++p) {
    const int blk = trl_checked(a.table[(size_t)seq * a.max_blocks + p], a.n_blocks, 15), keys = min(KVB, range.y - p * KVB);
    const T* kp = reinterpret_cast<const T*>(a.pages + ((size_t)blk * a.n_kv + kvh) * a.page_bytes);
    const T* vp = kp + KVB * dk;
    __syncthreads();
    for (int x = threadIdx.x; x < KVB * dk; x += 256) {
      const int kr = x / dk, d = x % dk;
      sk[kr * (dk + 1) + d] = kr < keys ? to_f(kp[(kr * kch + page_chunk(d / C, kr, kch)) * C + d % C]) : 0.f;
    }
    for (int x = threadIdx.x; x < KVB * dv; x += 256) {
      const int kr = x / dv, d = x % dv;
      sv[x] = kr < keys ? to_f(vp[(kr * vch + page_chunk(d / C, kr, vch)) * C + d % C]) : 0.f;
    }
    __syncthreads();
    float s = 0.f;
    for (int d = 0; d < dk; ++d) s = fmaf(sq[r * (dk + 1) + d], sk[c * (dk + 1) + d], s);
    s *= a.scale;
    if (a.cap > 0.f) s = a.cap * tanhf(s / a.cap);
    const int back = pos - (p * KVB + c);
    if (back < 0 || back >= win) s = -INFINITY;
    float top = s;
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));      // a row's 16 threads share half a warp
    top = fmaxf(top, m);
    const float ref = top == -INFINITY ? 0.f : top, f = m == -INFINITY ? 0.f : expf(m - ref), w = expf(s - ref);
    float ls = w;
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) ls += __shfl_xor_sync(0xffffffffu, ls, o);
    l = fmaf(l, f, ls), m = top;
    s_w[r][c] = w;
    __syncwarp();
#pragma unroll
    for (int i = 0; i < F_MAXD / 16; ++i) {
      const int d = c + 16 * i;
      if (d < dv) {
        acc[i] *= f;
#pragma unroll
        for (int j = 0; j < KVB; ++j) acc[i] = fmaf(s_w[r][j], sv[j * dv + d], acc[i]);
      }
    }
  }
  float g = 1.f;
  if (a.sink) {
    const float s = a.sink[h], top = fmaxf(m, s);
    g = expf(m - top), l = fmaf(l, g, expf(s - top));
  }
  g = in ? g / l * a.factor : 0.f;
  if (a.turn) {                                    // (uniform) a pair's halves meet where the values were
    __syncthreads();
    for (int i = 0; i < F_MAXD / 16; ++i)
      if (c + 16 * i < dv) sv[r * dv + c + 16 * i] = acc[i] * g;
    __syncwarp();                                  // a row's threads share a warp
    if (!in) return;
    for (int d = c; d < dv / 2; d += 16) {
      const float2 p = turn_back(sv[r * dv + d], sv[r * dv + dv / 2 + d], a.turn[(size_t)t * (dv / 2) + d]);
      T* out = reinterpret_cast<T*>(a.out) + (size_t)t * a.ldo + (size_t)h * dv + d;
      out[0] = from_f<T>(p.x), out[dv / 2] = from_f<T>(p.y);
    }
    return;
  }
  if (!in) return;
  for (int i = 0; i < F_MAXD / 16; ++i)
    if (c + 16 * i < dv) reinterpret_cast<T*>(a.out)[(size_t)t * a.ldo + (size_t)h * dv + c + 16 * i] = from_f<T>(acc[i] * g);
}

template <int D, int WM, int WN, bool FULL>
cudaError_t sm_launch_as(SmArgs a, int tiles, int B, const int* seq_ids, int n_tok, cudaStream_t st) {
  constexpr int ROWS = 16 * WM;
  const size_t q_bytes = (size_t)(ROWS * (a.kch * 16 + 16) + 127) / 128 * 128, stage = (size_t)TPAGES * a.page_bytes;
  const size_t room = WM == 1 ? 104 * 1024 : (size_t)SM_SMEM;   // decode blocks: two on an SM where three stages allow it
  int stages = 4;
  while (stages > 2 && q_bytes + stages * stage > room) --stages;
  if (WM == 1 && stages < 3 && q_bytes + 3 * stage <= (size_t)SM_SMEM) stages = 3;
  // the merge of WN warps, or rows to be turned, go through the ring
  const size_t merge = WN > 1 ? (size_t)WN * ROWS * a.vch * 32 : a.turn ? (size_t)ROWS * (a.vch * 32 + 32) : 0;
  const size_t smem = q_bytes + (stages * stage > merge ? stages * stage : merge);
  if (smem > (size_t)SM_SMEM) return cudaErrorInvalidValue;
  a.n_stages = stages;
  auto kern = sm_attn_kernel<D, WM, WN, FULL>;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SM_SMEM + 128);
    if (e != cudaSuccess) return e;
    cudaFuncSetAttribute(kern, cudaFuncAttributePreferredSharedMemoryCarveout, 100);
    cudaFuncSetAttribute(sm_combine_kernel, cudaFuncAttributePreferredSharedMemoryCarveout, 100);
    configured = true;
  }
  cudaError_t e = trl_launch(kern, dim3(tiles * a.n_splits, a.n_kv, B), dim3((WM * WN + 1) * 32), smem + 128, st, a);
  if (e == cudaSuccess && a.n_splits > 1)
    e = trl_launch(sm_combine_kernel, dim3(n_tok, a.n_q), dim3(CB_THREADS), 0, st, a, seq_ids, ROWS);
  return e;
}

template <int D, int WM, int WN>
cudaError_t sm_launch(const SmArgs& a, int tiles, int B, const int* seq_ids, int n_tok, cudaStream_t st) {
  if (a.kch == D / 8 && a.vch == D / 8) return sm_launch_as<D, WM, WN, true>(a, tiles, B, seq_ids, n_tok, st);
  return sm_launch_as<D, WM, WN, false>(a, tiles, B, seq_ids, n_tok, st);
}

}  // namespace

// args: a PrepArgs filled by the caller (tilerl_b200/ops/cuda_blocks.py mirrors it field by field).
TRL_API int trl_qkv_prep(const PrepArgs* args, int T, int f32, void* stream) {
  const PrepArgs& a = *args;
  const int per = f32 ? 4 : 8;
  const int widest = max(a.k0, a.n_in - a.k0);
  const size_t smem = (size_t)(widest + 2 * a.n_pairs + max(a.heads, a.kv_heads) + 2 + (a.vfreqs ? a.dv : 0)) * sizeof(float);
  if (T <= 0 || a.ldp % per || a.n_in % 16 || a.n_in > a.ldp || a.dk % 16 || a.dv % 16 || a.heads <= 0 || a.kv_heads <= 0 || a.dim > a.dk ||
      2 * a.n_pairs > a.dim || a.k0 != a.heads * a.dk || a.n_in != (a.own ? a.v0 + a.kv_heads * a.dv : a.k0) || smem > 200 * 1024 ||
      ((uintptr_t)a.proj & 15) || !a.q || (a.own && (!a.pages || !a.k_norm != !a.q_norm || ((uintptr_t)a.pages & 15))) ||
      (a.taps && (!a.conv || !a.ring || a.taps > a.ring_rows || a.ring_ld % per || a.ring_slot % per || ((uintptr_t)a.ring & 15))) ||
      (a.mid && (a.pad0 < 0 || a.pad0 > a.ldm)) || (a.vfreqs && (!a.turn || !a.own || a.v0 == a.k0)))
    return (int)cudaErrorInvalidValue;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(qkv_prep_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(qkv_prep_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const int threads = T <= 148 && widest >= 2048 ? 512 : (widest >= 1024 ? 256 : 128);
  const dim3 grid(T, a.own ? 2 : 1);
  if (f32) return (int)trl_launch(qkv_prep_kernel<float>, grid, dim3(threads), smem, (cudaStream_t)stream, a);
  return (int)trl_launch(qkv_prep_kernel<bf16>, grid, dim3(threads), smem, (cudaStream_t)stream, a);
}

// Rows of a wide row tile: 128, or 112 for the widest heads (a ninth warp would leave 168 registers a thread).
TRL_API int trl_softmax_attn_rows(int dk, int dv) { return (dk > dv ? dk : dv) > 128 ? 112 : 128; }
// Head widths that the tensor-core form takes.
TRL_API int trl_softmax_attn_ok(int dk, int dv) { return dk <= 256 && dv <= 256; }

// q: [T, n_q * dk]; out: [T, ldo], first n_q * dv columns, times factor.  window 0: all earlier keys; cap 0: none; sink: fp32 [n_q] or
// null.  Serves the sequences with min_len <= q_len <= max_len: wide = 0 in row tiles of 16 (key work split over four warps), wide = 1
// in row tiles of trl_softmax_attn_rows(dk, dv), wide = 2 on CUDA cores (any length, no splits).  tiles: row tiles of the longest such
// sequence.  turn: fp32 [T, dv / 2, 2] cos and sin by which finished rows are turned back, column d with d + dv / 2, or null.  part, ml: fp32 [T, n_q, n_splits, dv] and [T, n_q, n_splits, 2].
TRL_API int trl_softmax_attn(const void* q, const void* pages, int n_blocks, const void* table, int max_blocks, const void* q_start,
                             const void* q_len, const void* positions, const void* seq_ids, const void* sink, void* out, int ldo, void* part,
                             void* ml, int T, int B, int tiles, int min_len, int max_len, int n_q, int n_kv, int dk, int dv, int n_splits,
                             int wide, int window, float scale, float cap, float factor, const void* turn, int f32, void* stream) {
  const int per = f32 ? 4 : 8;
  if (T <= 0 || B <= 0 || tiles <= 0 || n_kv <= 0 || n_q % n_kv || dk % 16 || dv % 16 || dk > F_MAXD || dv > F_MAXD || dk <= 0 || dv <= 0 ||
      n_splits < 1 || n_splits > 64 || (n_splits > 1 && (!part || !ml)) || ldo % per || n_blocks <= 0 || window < 0 || cap < 0.f || ((uintptr_t)turn & 15) || ((uintptr_t)pages & 15) ||
      ((uintptr_t)q & 15) || ((uintptr_t)out & 15) || (wide != 2 && (f32 || dk > 256 || dv > 256)))
    return (int)cudaErrorInvalidValue;
  SmArgs a;
  a.q = q, a.pages = (const unsigned char*)pages, a.kch = dk / per, a.vch = dv / per, a.page_bytes = KVB * (a.kch + a.vch) * 16;
  a.n_blocks = n_blocks, a.table = (const int*)table, a.max_blocks = max_blocks;
  a.q_start = (const int*)q_start, a.q_len = (const int*)q_len, a.positions = (const int*)positions;
  a.sink = (const float*)sink, a.out = out, a.ldo = ldo, a.part = (float*)part, a.ml = (float2*)ml;
  a.n_q = n_q, a.n_kv = n_kv, a.n_splits = n_splits, a.n_stages = 2, a.window = window, a.min_len = min_len, a.max_len = max_len;
  a.scale = scale, a.cap = cap, a.factor = factor, a.turn = (const float2*)turn;
  cudaStream_t st = (cudaStream_t)stream;
  const int d = dk > dv ? dk : dv;
  const int* si = (const int*)seq_ids;
  if (wide == 2) {
    const size_t smem = (size_t)((F_ROWS + KVB) * (dk + 1) + KVB * dv) * sizeof(float);
    static bool configured = false;
    if (!configured) {
      cudaError_t e = cudaFuncSetAttribute(sm_attn_plain_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 112 * 1024);
      if (e == cudaSuccess) e = cudaFuncSetAttribute(sm_attn_plain_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 112 * 1024);
      if (e != cudaSuccess) return (int)e;
      configured = true;
    }
    const dim3 grid(tiles, n_kv, B);
    if (f32) return (int)trl_launch(sm_attn_plain_kernel<float>, grid, dim3(256), smem, st, a);
    return (int)trl_launch(sm_attn_plain_kernel<bf16>, grid, dim3(256), smem, st, a);
  }
  if (wide) {
    if (d <= 64) return (int)sm_launch<64, 8, 1>(a, tiles, B, si, T, st);
    if (d <= 128) return (int)sm_launch<128, 8, 1>(a, tiles, B, si, T, st);
    return (int)sm_launch<256, 7, 1>(a, tiles, B, si, T, st);
  }
  if (d <= 64) return (int)sm_launch<64, 1, 4>(a, tiles, B, si, T, st);
  if (d <= 128) return (int)sm_launch<128, 1, 4>(a, tiles, B, si, T, st);
  return (int)sm_launch<256, 1, 4>(a, tiles, B, si, T, st);
}
