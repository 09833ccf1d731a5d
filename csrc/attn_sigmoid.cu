// Causal attention whose weights are sigmoid(q.k * scale + bias[head]), not normalised over keys, on the packed
// paged pool (page layout: tilerl_b200/kv.py, KvPage).
//
// Queries and keys are RMS-normalised per head without a weight.  The norm is one factor per row, so neither is
// ever written back normalised: scores are formed from the projected bf16 values with fp32 accumulation and
// multiplied by the two fp32 factors (the key's lies in its page, the query's is computed here).  Weights keep
// fp32 precision into the value product as a bf16 pair (high part + rest): sums over thousands of keys whose
// weights are far below one would otherwise carry the rounding of every weight.
// Without a softmax there is no running maximum and no rescaling: key ranges are independent and partial
// results add up.
//
//   sig_attn_kernel<D, WM, WN>  tensor cores (mma.sync m16n8k16 bf16).  One block = (16 WM query rows, kv head,
//       sequence, key split); a row is a (token, head of the group) pair, so the G heads of a kv head share every
//       page.  Keys come 64 at a time (four pages) into a ring of stages, one bulk copy per page, from a producing
//       warp; WN warps share a row tile and own 4 / WN pages of every stage each.  <.., 1, 4> serves decoding and
//       short windows (up to 16 rows), <.., 8, 1> and <256, 7, 1> prompts.
//   sig_combine_kernel          adds the splits of a row.
//   sig_attn_f32_kernel         the same attention in fp32 (CUDA cores) on an fp32 pool.
//
// Reference parity: the reference's attention is softmax only (no counterpart).
#include "packed.cuh"

namespace {

constexpr int TILE = 64, TPAGES = TILE / KVB, RMS_BYTES = 128;
constexpr long long SA_WAIT_CYCLES = 4000000000LL;
constexpr int SA_SMEM = 216 * 1024;
constexpr float LOG2E = 1.4426950408889634f;

struct SigArgs {
  const bf16* q;                       // fused projection rows, query heads first
  int ldq;
  const unsigned char* pages;          // [n_blocks, n_kv, page_bytes]
  int page_bytes, kch, vch, n_blocks;  // 16-byte chunks of a K / V row
  const int* table;
  int max_blocks;
  const int *q_start, *q_len, *positions;
  const float* bias;
  bf16* out;
  int ldo;
  float* part;                         // [T, n_q, n_splits, vch * 8]
  int n_q, n_kv, n_splits, n_stages, dim, min_len, max_len;
  float eps, scale;
};

// Key range of a row tile: pages per split (a multiple of a stage) for the tile's key count.
__device__ __forceinline__ int split_pages(int kv_len, int n_splits) {
  const int pages = (kv_len + KVB - 1) / KVB;
  const int want = max(1, min(n_splits, (kv_len + 2 * TILE - 1) / (2 * TILE)));
  return ((pages + want - 1) / want + TPAGES - 1) / TPAGES * TPAGES;
}
// Splits that hold keys; with one, the block writes the output row itself and there is nothing to combine.
__device__ __forceinline__ int splits_used(int kv_len, int n_splits) {
  const int pages = (kv_len + KVB - 1) / KVB, pps = split_pages(kv_len, n_splits);
  return (pages + pps - 1) / pps;
}
// Keys the rows [row0, row0 + rows) of a sequence see.
__device__ __forceinline__ int tile_keys(int row0, int rows, int n_rows, int G, int q0, const int* positions) {
  return positions[q0 + (min(row0 + rows, n_rows) - 1) / G] + 1;
}

__device__ __forceinline__ uint32_t sa_try_wait(uint32_t bar, uint32_t parity) {
  uint32_t ok;
  asm volatile("{ .reg .pred p;\n"
               "  mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n"
               "  selp.u32 %0, 1, 0, p; }\n"
               : "=r"(ok) : "r"(bar), "r"(parity) : "memory");
  return ok;
}
// sigmoid of a score given as t = -log2(e) x: 1 / (1 + 2^t)
__device__ __forceinline__ float sigmoid_weight(float t) {
  float e, r;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(t));
  asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + e));
  return r;
}

// FULL: K and V rows are D wide, so every chunk place is a constant away from one of four addresses a thread keeps.
template <int D, int WM, int WN, bool FULL>
__global__ void __launch_bounds__((WM * WN + 1) * 32)
sig_attn_kernel(const SigArgs a) {
  constexpr int ROWS = 16 * WM, NP = TPAGES / WN, NWC = WM * WN, THREADS = (NWC + 1) * 32;
  extern __shared__ unsigned char sa_smem_raw[];
  __shared__ float s_q[ROWS];                              // query factor x scale
  __shared__ __align__(8) uint64_t s_bar[8];               // full[4], empty[4]
  __shared__ volatile int s_ok;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int kch = FULL ? D / 8 : a.kch, vch = FULL ? D / 8 : a.vch, page_bytes = FULL ? KVB * D * 4 + RMS_BYTES : a.page_bytes;
  const uint32_t raw_a = (uint32_t)__cvta_generic_to_shared(sa_smem_raw);
  unsigned char* sa_smem = sa_smem_raw + (((raw_a + 127u) & ~127u) - raw_a);
  const uint32_t bar_a = (uint32_t)__cvta_generic_to_shared(s_bar);
  if (threadIdx.x == 0) {
    for (int st = 0; st < a.n_stages; ++st) {
      asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(bar_a + 8u * st));
      asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar_a + 32u + 8u * st), "r"(NWC));
    }
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    s_ok = 1;
  }
  pdl_enter(25);
  pdl_wait();
  const int n_tiles_x = gridDim.x / a.n_splits;
  const int tile = n_tiles_x - 1 - (int)blockIdx.x / a.n_splits, split = blockIdx.x % a.n_splits;   // longest key ranges first
  const int kvh = blockIdx.y, seq = blockIdx.z;
  const int G = a.n_q / a.n_kv, T = a.q_len[seq], n_rows = T * G, row0 = tile * ROWS;
  if (T < a.min_len || T > a.max_len || row0 >= n_rows) return;
  const int q0 = a.q_start[seq];
  const int kv_len = tile_keys(row0, ROWS, n_rows, G, q0, a.positions);
  const int pps = split_pages(kv_len, a.n_splits), used = splits_used(kv_len, a.n_splits);
  if (split >= used) return;
  const int lo = split * pps * KVB, hi = min(kv_len, (split + 1) * pps * KVB);
  const int n_tiles = (hi - lo + TILE - 1) / TILE;
  const int qld = kch * 16 + 16;                          // Q row stride in bytes: an odd number of 16-byte units
  const uint32_t q_a = (uint32_t)__cvta_generic_to_shared(sa_smem);
  const int q_bytes = (ROWS * qld + 127) / 128 * 128, stage_bytes = TPAGES * page_bytes;
  unsigned char* ring = sa_smem + q_bytes;
  const uint32_t ring_a = q_a + q_bytes;
  const int v_off = KVB * kch * 16 + RMS_BYTES;

  // query rows as projected, and their norm factors
  for (int r = warp; r < ROWS; r += NWC + 1) {
    const int row = row0 + r;
    float ss = 0.f;
    const bf16* src = a.q + (size_t)(q0 + row / G) * a.ldq + (size_t)(kvh * G + row % G) * (kch * 8);
    for (int c = lane; c < kch; c += 32) {
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (row < n_rows) v = *reinterpret_cast<const uint4*>(src + c * 8);
      *reinterpret_cast<uint4*>(sa_smem + r * qld + c * 16) = v;
      const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float2 f = bf162_bits_to_f2(w[i]);
        ss += f.x * f.x + f.y * f.y;
      }
    }
    ss = warp_sum(ss);
    if (lane == 0) s_q[r] = a.scale / sqrtf(ss / (float)a.dim + a.eps);
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
    if (sa_try_wait(bar, parity)) return true;
    const long long t_begin = clock64();
    for (uint32_t it = 1; !sa_try_wait(bar, parity); ++it) {
      if ((it & 63) == 0) {
        if (!s_ok) return false;
        if (clock64() - t_begin > SA_WAIT_CYCLES) {
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

  if (warp == NWC) {
    // ---------------- producer ----------------
    const int* table = a.table + (size_t)seq * a.max_blocks;
    int st = 0;
    uint32_t ph = 0;
    for (int kt = 0; kt < n_tiles; ++kt) {
      if (kt >= a.n_stages && !bounded_wait(bar_a + 32u + 8u * st, ph ^ 1u, 510 + st)) break;
      const int j0 = lo + kt * TILE, n_pg = min(TPAGES, (hi - j0 + KVB - 1) / KVB);
      uint32_t bytes = 0;
      const unsigned char* src = nullptr;
      if (lane < n_pg) {
        const int p = j0 / KVB + lane, keys = min(KVB, hi - p * KVB);
        const int blk = trl_checked(table[p], a.n_blocks, 6);
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
    int pos[2];
    float qf[2], bs[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int r = r_lo + 8 * i, row = row0 + r;
      const bool in = row < n_rows;
      pos[i] = in ? a.positions[q0 + row / G] : -1;
      qf[i] = s_q[r] * -LOG2E;
      bs[i] = in ? a.bias[kvh * G + row % G] * -LOG2E : 0.f;
    }
    const int my_rows = min(16, n_rows - row0 - wm * 16);   // keys this warp's rows see
    const int my_hi = my_rows > 0 ? min(hi, a.positions[q0 + (row0 + wm * 16 + my_rows - 1) / G] + 1) : 0;
    const int my_lo = my_rows > 0 ? a.positions[q0 + (row0 + wm * 16) / G] : 0;       // the first of them sees keys <= my_lo
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
      if (!bounded_wait(bar_a + 8u * st, ph, 500 + st)) break;
      const int jw = lo + kt * TILE + wn * NP * KVB;        // first key of this warp's pages
      if (jw < my_hi) {
        const uint32_t base = ring_a + st * stage_bytes + wn * NP * page_bytes;
        const unsigned char* base_p = ring + st * stage_bytes + wn * NP * page_bytes;
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
        // ---- weights, and O += W V
#pragma unroll
        for (int p = 0; p < NP; ++p) {
          if (jw + p * KVB < my_hi) {
            const float* kf = reinterpret_cast<const float*>(base_p + p * page_bytes + KVB * kch * 16);
            const bool edge = jw + p * KVB + KVB - 1 > my_lo;   // some row does not see all of this page
            uint32_t wh[4], wl[4];
#pragma unroll
            for (int n8 = 0; n8 < 2; ++n8) {
              const int c = n8 * 8 + (lane & 3) * 2, j = jw + p * KVB + c;
              const float2 f = *reinterpret_cast<const float2*>(kf + c);
#pragma unroll
              for (int i = 0; i < 2; ++i) {
                float w0 = sigmoid_weight(fmaf(sc[p][n8][2 * i], qf[i] * f.x, bs[i]));
                float w1 = sigmoid_weight(fmaf(sc[p][n8][2 * i + 1], qf[i] * f.y, bs[i]));
                if (edge) {                                 // (a select: stale bytes past the range may be anything)
                  w0 = j <= pos[i] ? w0 : 0.f;
                  w1 = j + 1 <= pos[i] ? w1 : 0.f;
                }
                const uint32_t h = f2_to_bf162_bits(w0, w1);
                const float2 hf = bf162_bits_to_f2(h);
                wh[n8 * 2 + i] = h;
                wl[n8 * 2 + i] = f2_to_bf162_bits(w0 - hf.x, w1 - hf.y);
              }
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
  }
  __syncthreads();
  pdl_trigger();                                            // (not earlier: waiting blocks would take the room of working ones)
  if (!s_ok) {                                              // copies may still be in flight towards this block
    const long long t_begin = clock64();
    while (clock64() - t_begin < 2000000LL) {
    }
  }
  const int dv = vch * 8;
  auto dst_part = [&](int row) {
    const int t = q0 + row / G, h = kvh * G + row % G;
    return a.part + (((size_t)t * a.n_q + h) * a.n_splits + split) * dv;
  };
  auto dst_out = [&](int row) { return a.out + (size_t)(q0 + row / G) * a.ldo + (size_t)(kvh * G + row % G) * dv; };
  if constexpr (WN == 1) {
    if (warp == NWC) return;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int row = row0 + wm * 16 + (lane >> 2) + 8 * i;
      if (row >= n_rows) continue;
#pragma unroll
      for (int nd = 0; nd < D / 8; ++nd) {
        if (FULL || nd < vch) {
          const int d = nd * 8 + (lane & 3) * 2;
          if (used == 1) *reinterpret_cast<uint32_t*>(dst_out(row) + d) = f2_to_bf162_bits(o[nd][2 * i], o[nd][2 * i + 1]);
          else *reinterpret_cast<float2*>(dst_part(row) + d) = make_float2(o[nd][2 * i], o[nd][2 * i + 1]);
        }
      }
    }
  } else {
    // the WN warps of a row tile saw different keys: add them in order, through the (idle) ring
    float* so = reinterpret_cast<float*>(ring);             // [WN][ROWS][dv]
    if (warp < NWC) {
#pragma unroll
      for (int nd = 0; nd < D / 8; ++nd) {
        if (FULL || nd < vch) {
          const int d = nd * 8 + (lane & 3) * 2, r = wm * 16 + (lane >> 2);
          *reinterpret_cast<float2*>(so + ((size_t)wn * ROWS + r) * dv + d) = make_float2(o[nd][0], o[nd][1]);
          *reinterpret_cast<float2*>(so + ((size_t)wn * ROWS + r + 8) * dv + d) = make_float2(o[nd][2], o[nd][3]);
        }
      }
    }
    __syncthreads();
    const int rows = min(ROWS, n_rows - row0);
    for (int x = threadIdx.x; x < rows * dv; x += THREADS) {
      const int r = x / dv, d = x % dv;
      float v = 0.f;
#pragma unroll
      for (int k = 0; k < WN; ++k) v += so[((size_t)k * ROWS + r) * dv + d];
      if (used == 1) dst_out(row0 + r)[d] = __float2bfloat16(v);
      else dst_part(row0 + r)[d] = v;
    }
  }
}

// grid (token, head): adds the partial rows of a launch whose row tiles were `rows` tall
__global__ void __launch_bounds__(128) sig_combine_kernel(const SigArgs a, const int* seq_ids, int rows) {
  pdl_launch_dependents(26);
  pdl_wait();
  const int t = blockIdx.x, h = blockIdx.y, seq = seq_ids[t], T = a.q_len[seq];
  if (T < a.min_len || T > a.max_len) return;
  const int G = a.n_q / a.n_kv, q0 = a.q_start[seq];
  const int row0 = ((t - q0) * G + h % G) / rows * rows;
  const int used = splits_used(tile_keys(row0, rows, T * G, G, q0, a.positions), a.n_splits);
  if (used == 1) return;
  const int dv = a.vch * 8;
  const float* p = a.part + ((size_t)t * a.n_q + h) * a.n_splits * dv;
  for (int d = threadIdx.x * 2; d < dv; d += 256) {
    float2 v = make_float2(0.f, 0.f);
#pragma unroll 8
    for (int s = 0; s < used; ++s) {
      const float2 x = *reinterpret_cast<const float2*>(p + (size_t)s * dv + d);
      v.x += x.x, v.y += x.y;
    }
    *reinterpret_cast<uint32_t*>(a.out + (size_t)t * a.ldo + (size_t)h * dv + d) = f2_to_bf162_bits(v.x, v.y);
  }
}

// fp32: one block = (16 query rows, kv head, sequence), a page of keys at a time; thread (r, c) forms the score of
// row r and key c and owns the output columns c, c + 16, ... of row r.
constexpr int F_ROWS = 16, F_MAXD = 256;
__global__ void __launch_bounds__(256)
sig_attn_f32_kernel(const float* q, int ldq, const unsigned char* pages, int page_bytes, int kch, int vch, const int* table,
                    int max_blocks, int n_blocks, const int* q_start, const int* q_len, const int* positions,
                    const float* __restrict__ bias, float* out, int ldo, int n_q, int n_kv, int dim, float eps, float scale) {
  extern __shared__ float sf[];
  __shared__ float s_w[F_ROWS][KVB + 1], s_f[F_ROWS];
  pdl_launch_dependents(27);
  pdl_wait();
  const int kvh = blockIdx.y, seq = blockIdx.z, G = n_q / n_kv, T = q_len[seq], n_rows = T * G, row0 = blockIdx.x * F_ROWS;
  if (row0 >= n_rows) return;
  const int q0 = q_start[seq], dk = kch * 4, dv = vch * 4;
  float* sq = sf;                                  // [16][dk + 1]
  float* sk = sq + F_ROWS * (dk + 1);              // [16][dk + 1]
  float* sv = sk + KVB * (dk + 1);                 // [16][dv]
  const int r = threadIdx.x >> 4, c = threadIdx.x & 15, row = row0 + r;
  const bool in = row < n_rows;
  const int t = in ? q0 + row / G : q0, h = kvh * G + (in ? row % G : 0);
  float ss = 0.f;
  for (int d = c; d < dk; d += 16) {
    const float v = in ? q[(size_t)t * ldq + (size_t)h * dk + d] : 0.f;
    sq[r * (dk + 1) + d] = v;
    ss += v * v;
  }
#pragma unroll
  for (int o2 = 8; o2 > 0; o2 >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o2);
  const float qf = scale / sqrtf(ss / (float)dim + eps);
  const int pos = in ? positions[t] : -1;
  const float b = bias[h];
  float acc[F_MAXD / 16];
#pragma unroll
  for (int i = 0; i < F_MAXD / 16; ++i) acc[i] = 0.f;
  const int kv_len = tile_keys(row0, F_ROWS, n_rows, G, q0, positions);
  for (int p = 0; p * KVB < kv_len; ++p) {
    const int blk = trl_checked(table[(size_t)seq * max_blocks + p], n_blocks, 7), keys = min(KVB, kv_len - p * KVB);
    const unsigned char* page = pages + ((size_t)blk * n_kv + kvh) * page_bytes;
    const float* kp = reinterpret_cast<const float*>(page);
    const float* fp = kp + KVB * dk;
    const float* vp = fp + RMS_BYTES / 4;
    __syncthreads();
    for (int x = threadIdx.x; x < KVB * dk; x += 256) {
      const int kr = x / dk, d = x % dk;
      sk[kr * (dk + 1) + d] = kr < keys ? kp[(kr * kch + page_chunk(d / 4, kr, kch)) * 4 + d % 4] : 0.f;
    }
    for (int x = threadIdx.x; x < KVB * dv; x += 256) {
      const int kr = x / dv, d = x % dv;
      sv[x] = kr < keys ? vp[(kr * vch + page_chunk(d / 4, kr, vch)) * 4 + d % 4] : 0.f;
    }
    if (threadIdx.x < KVB) s_f[threadIdx.x] = threadIdx.x < keys ? fp[threadIdx.x] : 0.f;
    __syncthreads();
    float s = 0.f;
    for (int d = 0; d < dk; ++d) s = fmaf(sq[r * (dk + 1) + d], sk[c * (dk + 1) + d], s);
    s_w[r][c] = p * KVB + c <= pos ? 1.f / (1.f + expf(-(s * qf * s_f[c] + b))) : 0.f;
    __syncwarp();                                  // a row's 16 threads share a warp
#pragma unroll
    for (int i = 0; i < F_MAXD / 16; ++i) {
      const int d = c + 16 * i;
      if (d < dv) {
#pragma unroll
        for (int j = 0; j < KVB; ++j) acc[i] = fmaf(s_w[r][j], sv[j * dv + d], acc[i]);
      }
    }
  }
  if (in)
    for (int i = 0; i < F_MAXD / 16; ++i)
      if (c + 16 * i < dv) out[(size_t)t * ldo + (size_t)h * dv + c + 16 * i] = acc[i];
}

template <int D, int WM, int WN, bool FULL>
cudaError_t sig_launch_as(SigArgs a, int tiles, int B, const int* seq_ids, int n_tok, cudaStream_t st) {
  constexpr int ROWS = 16 * WM;
  const size_t q_bytes = (size_t)(ROWS * (a.kch * 16 + 16) + 127) / 128 * 128, stage = (size_t)TPAGES * a.page_bytes;
  const size_t room = WM == 1 ? 104 * 1024 : (size_t)SA_SMEM;   // decode blocks: two on an SM where three stages allow it
  int stages = 4;
  while (stages > 2 && q_bytes + stages * stage > room) --stages;
  if (WM == 1 && stages < 3 && q_bytes + 3 * stage <= (size_t)SA_SMEM) stages = 3;
  if (q_bytes + stages * stage > (size_t)SA_SMEM) return cudaErrorInvalidValue;
  a.n_stages = stages;
  auto kern = sig_attn_kernel<D, WM, WN, FULL>;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SA_SMEM + 128);
    if (e != cudaSuccess) return e;
    cudaFuncSetAttribute(kern, cudaFuncAttributePreferredSharedMemoryCarveout, 100);
    cudaFuncSetAttribute(sig_combine_kernel, cudaFuncAttributePreferredSharedMemoryCarveout, 100);
    configured = true;
  }
  cudaError_t e = trl_launch(kern, dim3(tiles * a.n_splits, a.n_kv, B), dim3((WM * WN + 1) * 32), q_bytes + stages * stage + 128, st, a);
  if (e == cudaSuccess && a.n_splits > 1)
    e = trl_launch(sig_combine_kernel, dim3(n_tok, a.n_q), dim3(128), 0, st, a, seq_ids, ROWS);
  return e;
}

template <int D, int WM, int WN>
cudaError_t sig_launch(const SigArgs& a, int tiles, int B, const int* seq_ids, int n_tok, cudaStream_t st) {
  if (a.kch == D / 8 && a.vch == D / 8) return sig_launch_as<D, WM, WN, true>(a, tiles, B, seq_ids, n_tok, st);
  return sig_launch_as<D, WM, WN, false>(a, tiles, B, seq_ids, n_tok, st);
}

}  // namespace

// Rows of a wide row tile: 128, or 112 for the widest heads (a ninth warp would leave 168 registers a thread).
TRL_API int trl_sigmoid_attn_rows(int dk, int dv) { return (dk > dv ? dk : dv) > 128 ? 112 : 128; }

// q: fused projection rows [T, ldq] whose first n_q * dk columns are the query heads; out: [T, ldo], first n_q * dv columns.
// Serves the sequences with min_len <= q_len <= max_len: wide = 0 in row tiles of 16 (key work split over four warps),
// wide = 1 in row tiles of
// trl_sigmoid_attn_rows(dk, dv).  tiles: row tiles of the longest such sequence.  part: fp32 [T, n_q, n_splits, dv].
TRL_API int trl_sigmoid_attn(const void* q, int ldq, const void* pages, int n_blocks, const void* table, int max_blocks,
                             const void* q_start, const void* q_len, const void* positions, const void* seq_ids,
                             const void* bias, void* out, int ldo, void* part, int T, int B, int tiles, int min_len, int max_len,
                             int n_q, int n_kv, int dim, int dk, int dv, int n_splits, int wide, float eps, float scale,
                             void* stream) {
  if (T <= 0 || B <= 0 || tiles <= 0 || n_kv <= 0 || n_q % n_kv || dk % 16 || dv % 16 || dk > 256 || dv > 256 || dk <= 0 ||
      dv <= 0 || dim <= 0 || dim > dk || n_splits < 1 || (n_splits > 1 && !part) || ldq % 8 || ldo % 8 || n_blocks <= 0 ||
      ((uintptr_t)pages & 15) || ((uintptr_t)q & 15) || ((uintptr_t)out & 15))
    return (int)cudaErrorInvalidValue;
  SigArgs a;
  a.q = (const bf16*)q, a.ldq = ldq, a.pages = (const unsigned char*)pages, a.kch = dk / 8, a.vch = dv / 8;
  a.page_bytes = KVB * (a.kch + a.vch) * 16 + RMS_BYTES, a.n_blocks = n_blocks;
  a.table = (const int*)table, a.max_blocks = max_blocks;
  a.q_start = (const int*)q_start, a.q_len = (const int*)q_len, a.positions = (const int*)positions;
  a.bias = (const float*)bias, a.out = (bf16*)out, a.ldo = ldo, a.part = (float*)part;
  a.n_q = n_q, a.n_kv = n_kv, a.n_splits = n_splits, a.n_stages = 2, a.dim = dim, a.min_len = min_len, a.max_len = max_len;
  a.eps = eps, a.scale = scale;
  cudaStream_t st = (cudaStream_t)stream;
  const int d = dk > dv ? dk : dv;
  const int* si = (const int*)seq_ids;
  if (wide) {
    if (d <= 64) return (int)sig_launch<64, 8, 1>(a, tiles, B, si, T, st);
    if (d <= 128) return (int)sig_launch<128, 8, 1>(a, tiles, B, si, T, st);
    return (int)sig_launch<256, 7, 1>(a, tiles, B, si, T, st);
  }
  if (d <= 64) return (int)sig_launch<64, 1, 4>(a, tiles, B, si, T, st);
  if (d <= 128) return (int)sig_launch<128, 1, 4>(a, tiles, B, si, T, st);
  return (int)sig_launch<256, 1, 4>(a, tiles, B, si, T, st);
}

// fp32 pool and activations; every sequence of the batch.
TRL_API int trl_sigmoid_attn_f32(const void* q, int ldq, const void* pages, int n_blocks, const void* table, int max_blocks,
                                 const void* q_start, const void* q_len, const void* positions, const void* bias, void* out,
                                 int ldo, int B, int max_q_len, int n_q, int n_kv, int dim, int dk, int dv, float eps,
                                 float scale, void* stream) {
  if (B <= 0 || max_q_len <= 0 || n_kv <= 0 || n_q % n_kv || dk % 16 || dv % 16 || dk > F_MAXD || dv > F_MAXD || dk <= 0 ||
      dv <= 0 || dim <= 0 || dim > dk || n_blocks <= 0)
    return (int)cudaErrorInvalidValue;
  const int kch = dk / 4, vch = dv / 4, page_bytes = KVB * (kch + vch) * 16 + RMS_BYTES;
  const size_t smem = (size_t)((F_ROWS + KVB) * (dk + 1) + KVB * dv) * sizeof(float);
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(sig_attn_f32_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 64 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const dim3 grid((max_q_len * (n_q / n_kv) + F_ROWS - 1) / F_ROWS, n_kv, B);
  return (int)trl_launch(sig_attn_f32_kernel, grid, dim3(256), smem, (cudaStream_t)stream, (const float*)q, ldq,
                         (const unsigned char*)pages, page_bytes, kch, vch, (const int*)table, max_blocks, n_blocks,
                         (const int*)q_start, (const int*)q_len, (const int*)positions, (const float*)bias, (float*)out, ldo,
                         n_q, n_kv, dim, eps, scale);
}
