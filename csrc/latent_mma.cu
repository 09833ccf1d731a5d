// Latent attention in bf16 on tensor cores (mma.sync), in its two forms.  Cache and symbols: latent.cu.
//
// Few query tokens (decoding, verify windows, short portions): queries are mapped into the latent and every head reads the
// same cached rows, so a page is fetched once for all heads.
//   latent_absorb_kernel  q W_uk per head, and the rotated part beside it: query rows [kv | rd] of every (token, head).
//   latent_decode_kernel  one block = 16 (token, head) rows of a sequence and a share of the window's keys.  Pages come
//                         through a ring of stages (one bulk copy each, from a producing warp).  Of a stage's 64 keys each of eight
//                         warps scores eight; every warp then forms all weights and sums an eighth of the latent's columns.
//   latent_out_kernel     merges the shares, maps the sum back (W_uv) and applies the output gate.
// Prompts: keys and values of the window are expanded once for all query tokens.
//   latent_gather_kernel  cached rows of a range of positions, dense; the expansion itself is one library product.
//   latent_prompt_kernel  windowed softmax attention per head, 128 query tokens x 64 keys, output gate in the epilogue.
//
// Scores, softmax and sums are fp32; weights enter the value product as a bf16 pair (value and rest).
// Reference parity: the reference's attention keeps full keys and values (no counterpart).
#include "packed.cuh"

namespace {

constexpr int TILE = 64, TPAGES = TILE / KVB;
constexpr long long LD_WAIT_CYCLES = 4000000000LL;
constexpr int LD_SMEM = 216 * 1024, MAX_SPLITS = 32;
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ bool in_class(int n, int lo, int hi) { return n >= lo && n <= hi; }

// acc += 16 weight rows x 8 token columns over K (a multiple of 16): wa, wb point at rows g and g + 8 of the tile (g = lane / 4)
// plus 8 (lane % 4); xs at token g's row of the activations in shared memory plus the same.  The 8 values a lane loads of a
// row serve two MMAs under a permutation of k that the activations share.
template <bool TWO>
__device__ __forceinline__ void rows16(float (&acc)[4], const bf16* __restrict__ wa, const bf16* __restrict__ wb, const bf16* xs, const bf16* xl,
                                       int K, int t4) {
#pragma unroll 4
  for (int k = 0; k < K; k += 32) {
    uint4 a = make_uint4(0u, 0u, 0u, 0u), b = a, x = a, y = a;
    if (k + t4 * 8 < K) {
      a = *reinterpret_cast<const uint4*>(wa + k), b = *reinterpret_cast<const uint4*>(wb + k);
      x = *reinterpret_cast<const uint4*>(xs + k);
      if (TWO) y = *reinterpret_cast<const uint4*>(xl + k);
    }
    const uint32_t f0[4] = {a.x, b.x, a.y, b.y}, f1[4] = {a.z, b.z, a.w, b.w};
    mma16(acc, f0, x.x, x.y);
    mma16(acc, f1, x.z, x.w);
    if (TWO) mma16(acc, f0, y.x, y.y), mma16(acc, f1, y.z, y.w);
  }
}

// grid (head, 128 latent columns, 8 tokens), 256 threads: a warp forms 16 columns of 8 tokens.  ukt: [heads][kv][dk].
__global__ void __launch_bounds__(256)
latent_absorb_kernel(const bf16* q, int dq, int dk, int rd, const bf16* __restrict__ ukt, int kv, const double* __restrict__ freqs, int n_pairs,
                     float amp, const int* positions, const int* seq_ids, const int* q_len, int max_len, bf16* ql, int T, int heads) {
  extern __shared__ __align__(16) unsigned char ab_raw[];
  __shared__ bf16 s_o[8][128];
  bf16* xs = reinterpret_cast<bf16*>(ab_raw);            // [8][dk + 8]
  pdl_launch_dependents(44);
  const int h = blockIdx.x, c0 = blockIdx.y * 128, t0 = blockIdx.z * 8, n = min(8, T - t0), tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const int ldx = dk + 8, D = kv + rd;
  pdl_wait();
  const bool in = tid < n && q_len[seq_ids[t0 + tid]] <= max_len;
  if (!__syncthreads_or(in)) return;
  for (int x = tid; x < 8 * (dk / 8); x += 256) {
    const int t = x / (dk / 8), c = x % (dk / 8);
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (t < n) v = *reinterpret_cast<const uint4*>(q + ((size_t)(t0 + t) * heads + h) * dq + c * 8);
    *reinterpret_cast<uint4*>(xs + t * ldx + c * 8) = v;
  }
  if (blockIdx.y == 0)                                   // the rotated part, turned unless it already is (n_pairs 0)
    for (int x = tid; x < n * (rd / 2); x += 256) {
      const int t = x / (rd / 2), p = x % (rd / 2);
      float2 v = bf162_bits_to_f2(*reinterpret_cast<const uint32_t*>(q + ((size_t)(t0 + t) * heads + h) * dq + dk + 2 * p));
      if (p < n_pairs) {
        float cs, sn;
        pair_angle(positions[t0 + t], freqs[p], amp, cs, sn);
        v = make_float2(v.x * cs - v.y * sn, v.y * cs + v.x * sn);
      }
      *reinterpret_cast<uint32_t*>(ql + ((size_t)(t0 + t) * heads + h) * D + kv + 2 * p) = f2_to_bf162_bits(v.x, v.y);
    }
  __syncthreads();
  const int g = lane >> 2, t4 = lane & 3, r0 = c0 + warp * 16;
  float acc[4] = {0.f, 0.f, 0.f, 0.f};
  if (r0 < kv) {                                         // (kv is a multiple of 16)
    const bf16* w = ukt + ((size_t)h * kv + r0 + g) * dk + t4 * 8;
    rows16<false>(acc, w, w + (size_t)8 * dk, xs + g * ldx + t4 * 8, nullptr, dk, t4);
  }
#pragma unroll
  for (int e = 0; e < 4; ++e) s_o[2 * t4 + (e & 1)][warp * 16 + g + (e >> 1) * 8] = __float2bfloat16(acc[e]);
  __syncthreads();
  for (int x = tid; x < n * 16; x += 256) {
    const int t = x >> 4, c = (x & 15) * 8;
    if (c0 + c < kv)
      *reinterpret_cast<uint4*>(ql + ((size_t)(t0 + t) * heads + h) * D + c0 + c) = *reinterpret_cast<const uint4*>(&s_o[t][c]);
  }
}

struct DecArgs {
  const bf16* ql;                      // [T, heads, kv + rd]
  const unsigned char* pages;
  int kch, vch, n_blocks;              // 16-byte chunks of a cached row, of its latent part
  const int* table;
  int max_blocks;
  const int *q_start, *q_len, *positions;
  float* part;                         // [T, heads, n_splits, kv]
  float2* ml;                          // [T, heads, n_splits]: running maximum (log2), sum
  int heads, n_splits, n_stages, window, min_len, max_len;
  float scale2;                        // scale x log2(e)
};

// First page and number of stages of a row tile's keys, and the stages of one split.
__device__ __forceinline__ void tile_range(int p_first, int p_last, int window, int& page0, int& stages) {
  page0 = max(0, p_first - window + 1) / KVB;
  stages = (p_last / KVB - page0) / TPAGES + 1;
}
__device__ __forceinline__ int stages_per_split(int stages, int n_splits) {
  const int want = max(1, min(n_splits, stages));
  return (stages + want - 1) / want;
}
__device__ __forceinline__ uint32_t ld_try_wait(uint32_t bar, uint32_t parity) {
  uint32_t ok;
  asm volatile("{ .reg .pred p;\n"
               "  mbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2;\n"
               "  selp.u32 %0, 1, 0, p; }\n"
               : "=r"(ok) : "r"(bar), "r"(parity) : "memory");
  return ok;
}

template <int CW>
__global__ void __launch_bounds__(288) latent_decode_kernel(const DecArgs a) {
  constexpr int NW = 8, SX = 72, THREADS = (NW + 1) * 32;
  extern __shared__ unsigned char ld_raw[];
  __shared__ __align__(8) uint64_t s_bar[9];               // full[4], empty[4], scores
  __shared__ __align__(16) float s_x[2][16][SX];           // scores of a stage's 64 keys
  __shared__ volatile int s_ok;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const uint32_t raw_a = (uint32_t)__cvta_generic_to_shared(ld_raw);
  unsigned char* smem = ld_raw + (((raw_a + 127u) & ~127u) - raw_a);
  const uint32_t smem_a = (raw_a + 127u) & ~127u, bar_a = (uint32_t)__cvta_generic_to_shared(s_bar);
  if (threadIdx.x == 0) {
    for (int st = 0; st < a.n_stages; ++st) {
      asm volatile("mbarrier.init.shared::cta.b64 [%0], 1;" ::"r"(bar_a + 8u * st));
      asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar_a + 32u + 8u * st), "r"(NW));
    }
    asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar_a + 64u), "r"(NW));
    asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    s_ok = 1;
  }
  pdl_enter(45);
  pdl_wait();
  const int tile = blockIdx.x / a.n_splits, split = blockIdx.x % a.n_splits, seq = blockIdx.y;
  const int T = a.q_len[seq], n_rows = T * a.heads, row0 = tile * 16;
  if (!in_class(T, a.min_len, a.max_len) || row0 >= n_rows) return;
  const int q0 = a.q_start[seq], rows = min(16, n_rows - row0);
  const int p_first = a.positions[q0 + row0 / a.heads], p_last = a.positions[q0 + (row0 + rows - 1) / a.heads];
  int page0, stages;
  tile_range(p_first, p_last, a.window, page0, stages);
  const int sps = stages_per_split(stages, a.n_splits);
  const int s0 = split * sps, s1 = min(stages, s0 + sps);
  if (s0 >= s1) return;
  const int row_b = a.kch * 16, page_b = KVB * row_b, stage_b = TPAGES * page_b, qld = row_b + 16;
  const int kv = a.vch * 8, D = a.kch * 8;
  const int q_bytes = (16 * qld + 127) / 128 * 128;
  unsigned char* ring = smem + q_bytes;
  const uint32_t ring_a = smem_a + q_bytes;
  const int lo = (page0 + s0 * TPAGES) * KVB, hi = min(p_last + 1, (page0 + s1 * TPAGES) * KVB);
  for (int x = threadIdx.x; x < 16 * a.kch; x += THREADS) {
    const int r = x / a.kch, c = x % a.kch, row = row0 + r;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (r < rows) v = *reinterpret_cast<const uint4*>(a.ql + ((size_t)(q0 + row / a.heads) * a.heads + row % a.heads) * D + c * 8);
    *reinterpret_cast<uint4*>(smem + r * qld + c * 16) = v;
  }
  {
    // The last page brings only the rows that exist (the pool may hold anything past them, and 0 x row must be 0): if
    // nothing was copied into that place before, its tail starts as zeros.
    const int last = s1 - s0 - 1, tail = hi & (KVB - 1);
    if (tail && last < a.n_stages) {
      const int pg = ((hi - 1 - lo) / KVB) % TPAGES;
      unsigned char* p = ring + last * stage_b + pg * page_b;
      for (int x = tail * a.kch + threadIdx.x; x < KVB * a.kch; x += THREADS) *reinterpret_cast<uint4*>(p + x * 16) = make_uint4(0u, 0u, 0u, 0u);
    }
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  }
  __syncthreads();
  auto bounded_wait = [&](uint32_t bar, uint32_t parity, int what) {
    if (ld_try_wait(bar, parity)) return true;
    const long long t_begin = clock64();
    for (uint32_t it = 1; !ld_try_wait(bar, parity); ++it) {
      if ((it & 63) == 0) {
        if (!s_ok) return false;
        if (clock64() - t_begin > LD_WAIT_CYCLES) {
          trl_set_error(TRL_ERR_MBAR_TIMEOUT, (int)blockIdx.x, what, (int)parity);
          s_ok = 0;
          return false;
        }
      }
    }
    return true;
  };
  float o[CW / 8][4], mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < CW / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  if (warp == NW) {
    // ---------------- producer ----------------
    const int* table = a.table + (size_t)seq * a.max_blocks;
    int st = 0;
    uint32_t ph = 0;
    for (int k = s0; k < s1; ++k) {
      if (k - s0 >= a.n_stages && !bounded_wait(bar_a + 32u + 8u * st, ph ^ 1u, 530 + st)) break;
      const int j0 = (page0 + k * TPAGES) * KVB, n_pg = min(TPAGES, (hi - j0 + KVB - 1) / KVB);
      uint32_t bytes = 0;
      const unsigned char* src = nullptr;
      if (lane < n_pg) {
        const int p = j0 / KVB + lane;
        src = a.pages + (size_t)trl_checked(table[p], a.n_blocks, 11) * page_b;
        bytes = (uint32_t)(min(KVB, hi - p * KVB) * row_b);
      }
      const uint32_t total = __reduce_add_sync(0xffffffffu, bytes), full = bar_a + 8u * st;
      if (lane == 0) asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(full), "r"(total) : "memory");
      __syncwarp();
      if (lane < n_pg)
        asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                     ::"r"(ring_a + st * stage_b + lane * page_b), "l"(src), "r"(bytes), "r"(full) : "memory");
      if (++st == a.n_stages) st = 0, ph ^= 1u;
    }
  } else {
    // ---------------- consumers ----------------
    int pos[2];
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int r = (lane >> 2) + 8 * i;
      pos[i] = r < rows ? a.positions[q0 + (row0 + r) / a.heads] : -1;
    }
    const uint32_t qa = smem_a + ((lane & 7) + ((lane >> 3) & 1) * 8) * qld + (lane >> 4) * 16;
    const int vr = (lane & 7) + ((lane >> 3) & 1) * 8, vcl = lane >> 4;
    const int page = warp >> 1, r8 = (warp & 1) * 8 + (lane & 7), c8 = lane >> 3;      // this warp scores 8 keys of a page
    const int nc = a.kch, rot8 = r8 % nc, vrot = vr % nc, g = lane >> 2, t4 = lane & 3;
    const bool xored = nc % 8 == 0;
    auto place = [&](int c, int r, int rot) {              // page_chunk without a division (rot = r % nc)
      const int x = c + rot;
      return xored ? c ^ (r & 7) : (x >= nc ? x - nc : x);
    };
    const int vc0 = warp * (CW / 8), vch = min(CW / 8, a.vch - vc0);      // this warp's output chunks (none: it only scores)
    int st = 0;
    uint32_t ph = 0, xp = 0;                               // xp: parity and buffer of the scores
    for (int k = s0; k < s1; ++k) {
      if (!bounded_wait(bar_a + 8u * st, ph, 520 + st)) break;
      const int j0 = (page0 + k * TPAGES) * KVB;
      const uint32_t stage = ring_a + st * stage_b;
      if (j0 + page * KVB < hi) {
        const uint32_t base = stage + page * page_b + r8 * row_b;
        float sc[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i) sc[i][0] = sc[i][1] = sc[i][2] = sc[i][3] = 0.f;
        int kk = 0;                                        // groups of 4 chunks: two k-steps
#pragma unroll 2
        for (; kk + 2 <= nc / 4; kk += 2) {
          uint32_t q[4][4], b[2][4];
          ldsm4(b[0], base + place(kk * 4 + c8, r8, rot8) * 16);
          ldsm4(b[1], base + place(kk * 4 + 4 + c8, r8, rot8) * 16);
#pragma unroll
          for (int i = 0; i < 4; ++i) ldsm4(q[i], qa + kk * 64 + i * 32);
#pragma unroll
          for (int i = 0; i < 4; ++i) mma16(sc[i], q[i], b[i >> 1][(i & 1) * 2], b[i >> 1][(i & 1) * 2 + 1]);
        }
        for (int c = kk * 4; c < nc; c += 2) {             // what is left, k-step by k-step
          uint32_t q[4], b[4];
          ldsm4(q, qa + c * 16);
          ldsm4(b, base + place(c + (c8 & 1), r8, rot8) * 16);
          mma16(sc[0], q, b[0], b[1]);
        }
        float* dst = &s_x[xp][g][warp * 8 + 2 * t4];
        *reinterpret_cast<float2*>(dst) = make_float2((sc[0][0] + sc[1][0]) + (sc[2][0] + sc[3][0]), (sc[0][1] + sc[1][1]) + (sc[2][1] + sc[3][1]));
        *reinterpret_cast<float2*>(dst + 8 * SX) = make_float2((sc[0][2] + sc[1][2]) + (sc[2][2] + sc[3][2]), (sc[0][3] + sc[1][3]) + (sc[2][3] + sc[3][3]));
      }
      __syncwarp();
      if (lane == 0) asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar_a + 64u) : "memory");
      if (!bounded_wait(bar_a + 64u, xp, 540)) break;
      // every warp forms the weights of all 64 keys (it needs them as operands), then sums its columns
      float w[TPAGES][2][4], back[2];
      bool moved = false;
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        float m = -INFINITY;
#pragma unroll
        for (int p = 0; p < TPAGES; ++p)
#pragma unroll
          for (int n8 = 0; n8 < 2; ++n8) {
            const float2 v = *reinterpret_cast<const float2*>(&s_x[xp][g + 8 * i][p * 16 + n8 * 8 + 2 * t4]);
            const int j = j0 + p * 16 + n8 * 8 + 2 * t4;   // (selects: scores past the range may be anything)
            w[p][n8][2 * i] = j <= pos[i] && pos[i] - j < a.window ? v.x * a.scale2 : -INFINITY;
            w[p][n8][2 * i + 1] = j + 1 <= pos[i] && pos[i] - j - 1 < a.window ? v.y * a.scale2 : -INFINITY;
            m = fmaxf(m, fmaxf(w[p][n8][2 * i], w[p][n8][2 * i + 1]));
          }
        m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 1));
        m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 2));
        const float now = fmaxf(mx[i], m), ref = now == -INFINITY ? 0.f : now;
        moved |= now > mx[i];
        back[i] = exp2f(mx[i] - ref);
        mx[i] = now;
        float ws = 0.f;
#pragma unroll
        for (int p = 0; p < TPAGES; ++p)
#pragma unroll
          for (int n8 = 0; n8 < 2; ++n8)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
              float& x = w[p][n8][2 * i + e];
              x = exp2f(x - ref);
              ws += x;
            }
        sum[i] = sum[i] * back[i] + ws;                    // (this lane's keys; added over the quad at the end)
      }
      xp ^= 1u;
      if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
        for (int nd = 0; nd < CW / 8; ++nd) o[nd][0] *= back[0], o[nd][1] *= back[0], o[nd][2] *= back[1], o[nd][3] *= back[1];
      }
#pragma unroll
      for (int p = 0; p < TPAGES; ++p) {
        if (j0 + p * KVB < hi) {
          uint32_t wh[4], wl[4];
#pragma unroll
          for (int n8 = 0; n8 < 2; ++n8)
#pragma unroll
            for (int i = 0; i < 2; ++i) split2(w[p][n8][2 * i], w[p][n8][2 * i + 1], wh[n8 * 2 + i], wl[n8 * 2 + i]);
#pragma unroll
          for (int nd = 0; nd < CW / 8; nd += 2) {
            if (nd < vch) {
              uint32_t b[4];
              ldsm4t(b, stage + p * page_b + (vr * nc + place(vc0 + nd + vcl, vr, vrot)) * 16);
              mma16(o[nd], wh, b[0], b[1]);
              mma16(o[nd + 1], wh, b[2], b[3]);
              mma16(o[nd], wl, b[0], b[1]);
              mma16(o[nd + 1], wl, b[2], b[3]);
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
      const int r = g + 8 * i, row = row0 + r;
      if (r >= rows) continue;
      const size_t at = ((size_t)(q0 + row / a.heads) * a.heads + row % a.heads) * a.n_splits + split;
      if (warp == 0 && t4 == 0) a.ml[at] = make_float2(mx[i], sum[i]);
#pragma unroll
      for (int nd = 0; nd < CW / 8; ++nd)
        if (nd < vch) *reinterpret_cast<float2*>(a.part + at * kv + (vc0 + nd) * 8 + 2 * t4) = make_float2(o[nd][2 * i], o[nd][2 * i + 1]);
    }
  }
  __syncthreads();
  pdl_trigger();
  if (!s_ok) {                                              // copies may still be in flight towards this block
    const long long t_begin = clock64();
    while (clock64() - t_begin < 2000000LL) {
    }
  }
}

// grid (head, 8 tokens, shares of the value rows), 256 threads
__global__ void __launch_bounds__(256)
latent_out_kernel(const float* part, const float2* ml, int n_splits, const bf16* __restrict__ uv, int kv, int dv, const bf16* gate, int ldp,
                  bf16* out, int n_out, const int* seq_ids, const int* q_start, const int* q_len, const int* positions, int T, int heads,
                  int window, int max_len) {
  extern __shared__ __align__(16) unsigned char oc_raw[];
  __shared__ float s_f[8][MAX_SPLITS];                   // factor of every share
  __shared__ int s_used[8];                              // shares of a token's row; 0: not this launch's
  const int ldx = kv + 8;
  bf16 *hi = reinterpret_cast<bf16*>(oc_raw), *lo = hi + 8 * ldx;       // [8][kv + 8] each
  pdl_launch_dependents(46);
  pdl_wait();
  const int h = blockIdx.x, t0 = blockIdx.y * 8, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  {
    const int t = t0 + warp;                             // a warp per token: maxima and sums of its shares
    int used = 0;
    if (t < T) {
      const int seq = seq_ids[t], len = q_len[seq], q0 = q_start[seq];
      if (len <= max_len && t - q0 < len) {
        const int n_rows = len * heads, row0 = ((t - q0) * heads + h) / 16 * 16;
        int page0, stages;
        tile_range(positions[q0 + row0 / heads], positions[q0 + (min(row0 + 16, n_rows) - 1) / heads], window, page0, stages);
        const int sps = stages_per_split(stages, n_splits);
        used = (stages + sps - 1) / sps;
        const size_t at = ((size_t)t * heads + h) * n_splits;
        const float2 v = lane < used ? ml[at + lane] : make_float2(-INFINITY, 0.f);
        const float m = warp_max(v.x), f = exp2f(v.x - m), l = warp_sum(f * v.y);
        if (lane < used) s_f[warp][lane] = f / l;
      }
    }
    if (lane == 0) s_used[warp] = used;
    if (!__syncthreads_or(used > 0)) return;
  }
  for (int x = tid; x < 8 * (kv / 4); x += 256) {
    const int t = x / (kv / 4), d = x % (kv / 4) * 4, used = s_used[t];
    const float* p = part + ((size_t)(t0 + t) * heads + h) * n_splits * kv + d;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int s = 0; s < used; ++s) {
      const float f = s_f[t][s];
      const float4 y = *reinterpret_cast<const float4*>(p + (size_t)s * kv);
      v.x = fmaf(f, y.x, v.x), v.y = fmaf(f, y.y, v.y), v.z = fmaf(f, y.z, v.z), v.w = fmaf(f, y.w, v.w);
    }
    uint2 a, b;
    split2(v.x, v.y, a.x, b.x), split2(v.z, v.w, a.y, b.y);
    *reinterpret_cast<uint2*>(hi + t * ldx + d) = a;
    *reinterpret_cast<uint2*>(lo + t * ldx + d) = b;
  }
  __syncthreads();
  const int g = lane >> 2, t4 = lane & 3;
  for (int tile = blockIdx.z * 8 + warp; tile * 16 < dv; tile += gridDim.z * 8) {
    float acc[4] = {0.f, 0.f, 0.f, 0.f};
    const bf16* w = uv + ((size_t)h * dv + tile * 16 + g) * kv + t4 * 8;
    rows16<true>(acc, w, w + (size_t)8 * kv, hi + g * ldx + t4 * 8, lo + g * ldx + t4 * 8, kv, t4);
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int t = 2 * t4 + (e & 1), d = h * dv + tile * 16 + g + (e >> 1) * 8;
      if (s_used[t])
        out[(size_t)(t0 + t) * n_out + d] = __float2bfloat16(acc[e] * sigmoid_x(__bfloat162float(gate[(size_t)(t0 + t) * ldp + d])));
    }
  }
  if (h == 0 && blockIdx.z == 0)
    for (int i = 0; i < 8; ++i)
      if (s_used[i])
        for (int c = heads * dv + tid; c < n_out; c += 256) out[(size_t)(t0 + i) * n_out + c] = __float2bfloat16(0.f);
}

// grid (positions lo .. of one sequence): cached rows -> c [n, kv], kr [n, rd]
__global__ void __launch_bounds__(64)
latent_gather_kernel(const unsigned char* pages, int n_blocks, const int* table, int lo, int kch, int vch, bf16* c, bf16* kr) {
  pdl_launch_dependents(47);
  pdl_wait();
  const int j = lo + blockIdx.x, r = j % KVB;
  const uint4* row = reinterpret_cast<const uint4*>(pages + (size_t)trl_checked(table[j / KVB], n_blocks, 12) * KVB * kch * 16) + r * kch;
  uint4* cd = reinterpret_cast<uint4*>(c) + (size_t)blockIdx.x * vch;
  uint4* kd = reinterpret_cast<uint4*>(kr) + (size_t)blockIdx.x * (kch - vch);
  for (int x = threadIdx.x; x < kch; x += 64) {
    const uint4 v = row[page_chunk(x, r, kch)];
    if (x < vch) cd[x] = v;
    else kd[x - vch] = v;
  }
}

struct PromptArgs {
  const bf16 *q, *kvx, *kr, *gate;     // query heads [T, heads, dq]; expanded [keys, ldkv]: heads x dk, heads x dv; [keys, rd]
  bf16* out;
  const int* positions;                // of the sequence's first query token on
  int n, lo, n_keys, heads, dq, dk, rd, dv, ldkv, ldp, n_out, window;
  float scale2;
};

// one block = (128 query tokens, head); a warp owns 16 of them
template <int DQ, int DV>
__global__ void __launch_bounds__(256) latent_prompt_kernel(const PromptArgs a) {
  constexpr int QROW = DQ * 2, VROW = DV * 2;
  extern __shared__ unsigned char lp_raw[];
  const uint32_t raw_a = (uint32_t)__cvta_generic_to_shared(lp_raw), q_a = (raw_a + 127u) & ~127u;
  const uint32_t k_a = q_a + 128 * QROW, v_a = k_a + 2 * TILE * QROW;
  pdl_launch_dependents(48);
  pdl_wait();
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, row0 = blockIdx.x * 128;
  const int rows = min(128, a.n - row0);
  auto off = [](int r, int c, int rowb) { return (uint32_t)(r * rowb + ((c ^ (r & 7)) << 4)); };
  auto zcp = [](uint32_t dst, const void* src, bool in) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(in ? 16 : 0) : "memory");
  };
  const int first = a.positions[row0], last = a.positions[row0 + rows - 1];
  const int j_lo = max(a.lo, first - a.window + 1), n_tiles = (last - j_lo) / TILE + 1;
  for (int x = tid; x < 128 * (DQ / 8); x += 256) {
    const int r = x / (DQ / 8), c = x % (DQ / 8);
    const bool in = r < rows && c * 8 < a.dq;
    zcp(q_a + off(r, c, QROW), a.q + (in ? ((size_t)(row0 + r) * a.heads + h) * a.dq + c * 8 : 0), in);
  }
  auto stage = [&](int kt, int b) {
    const int j0 = j_lo + kt * TILE - a.lo;                 // row of the expanded keys
    for (int x = tid; x < TILE * (DQ / 8); x += 256) {
      const int r = x / (DQ / 8), c = x % (DQ / 8);
      const bool in = j0 + r < a.n_keys && c * 8 < a.dq;
      const bf16* src = c * 8 < a.dk ? a.kvx + (size_t)(in ? j0 + r : 0) * a.ldkv + h * a.dk + c * 8
                                     : a.kr + (in ? (size_t)(j0 + r) * a.rd + c * 8 - a.dk : 0);
      zcp(k_a + b * TILE * QROW + off(r, c, QROW), src, in);
    }
    for (int x = tid; x < TILE * (DV / 8); x += 256) {
      const int r = x / (DV / 8), c = x % (DV / 8);
      const bool in = j0 + r < a.n_keys && c * 8 < a.dv;
      zcp(v_a + b * TILE * VROW + off(r, c, VROW), a.kvx + (in ? (size_t)(j0 + r) * a.ldkv + a.heads * a.dk + h * a.dv + c * 8 : 0), in);
    }
    cp_commit();
  };
  stage(0, 0);
  float o[DV / 8][4], mx[2] = {-INFINITY, -INFINITY}, sum[2] = {0.f, 0.f};
#pragma unroll
  for (int i = 0; i < DV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
  int pos[2];
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const int r = warp * 16 + (lane >> 2) + 8 * i;
    pos[i] = r < rows ? a.positions[row0 + r] : -1;
  }
  const bool live = warp * 16 < rows;
  const int w_first = live ? a.positions[row0 + warp * 16] : 0, w_last = live ? a.positions[row0 + min(rows, warp * 16 + 16) - 1] : -1;
  const int lrow = (lane & 7) + ((lane >> 3) & 1) * 8, lch = lane >> 4, brow = (lane & 7) + (lane >> 4) * 8, bch = (lane >> 3) & 1;
  const int nk = a.dq / 16, nv = a.dv / 8;
  for (int kt = 0; kt < n_tiles; ++kt) {
    const int b = kt & 1;
    cp_wait<0>();
    __syncthreads();                                        // tile kt is in, the other buffer is free
    if (kt + 1 < n_tiles) stage(kt + 1, b ^ 1);
    const int j0 = j_lo + kt * TILE;
    if (j0 > w_last || j0 + TILE - 1 <= w_first - a.window) continue;
    float sc[4][2][4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int n8 = 0; n8 < 2; ++n8) sc[j][n8][0] = sc[j][n8][1] = sc[j][n8][2] = sc[j][n8][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < DQ / 16; ++kk) {
      if (kk < nk) {
        uint32_t qf[4];
        ldsm4(qf, q_a + off(warp * 16 + lrow, kk * 2 + lch, QROW));
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          uint32_t kf[4];
          ldsm4(kf, k_a + b * TILE * QROW + off(16 * j + brow, kk * 2 + bch, QROW));
          mma16(sc[j][0], qf, kf[0], kf[1]);
          mma16(sc[j][1], qf, kf[2], kf[3]);
        }
      }
    }
    const bool edge = j0 + TILE - 1 > w_first || j0 <= w_last - a.window;      // some row does not see all of this tile
    float back[2];
    bool moved = false;
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      float m = -INFINITY;
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int n8 = 0; n8 < 2; ++n8)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            float& s = sc[j][n8][2 * i + e];
            s *= a.scale2;
            if (edge) {
              const int key = j0 + 16 * j + 8 * n8 + (lane & 3) * 2 + e;
              s = key <= pos[i] && pos[i] - key < a.window ? s : -INFINITY;
            }
            m = fmaxf(m, s);
          }
      m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 1));
      m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, 2));
      const float now = fmaxf(mx[i], m), ref = now == -INFINITY ? 0.f : now;
      moved |= now > mx[i];
      back[i] = exp2f(mx[i] - ref);
      mx[i] = now;
      float ws = 0.f;
#pragma unroll
      for (int j = 0; j < 4; ++j)
#pragma unroll
        for (int n8 = 0; n8 < 2; ++n8)
#pragma unroll
          for (int e = 0; e < 2; ++e) {
            float& s = sc[j][n8][2 * i + e];
            s = exp2f(s - ref);
            ws += s;
          }
      sum[i] = sum[i] * back[i] + ws;
    }
    if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
      for (int nd = 0; nd < DV / 8; ++nd) o[nd][0] *= back[0], o[nd][1] *= back[0], o[nd][2] *= back[1], o[nd][3] *= back[1];
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      uint32_t wh[4], wl[4];
#pragma unroll
      for (int n8 = 0; n8 < 2; ++n8)
#pragma unroll
        for (int i = 0; i < 2; ++i) split2(sc[j][n8][2 * i], sc[j][n8][2 * i + 1], wh[n8 * 2 + i], wl[n8 * 2 + i]);
#pragma unroll
      for (int nd = 0; nd < DV / 8; nd += 2) {
        if (nd < nv) {
          uint32_t f[4];
          ldsm4t(f, v_a + b * TILE * VROW + off(16 * j + lrow, nd + lch, VROW));
          mma16(o[nd], wh, f[0], f[1]);
          mma16(o[nd + 1], wh, f[2], f[3]);
          mma16(o[nd], wl, f[0], f[1]);
          mma16(o[nd + 1], wl, f[2], f[3]);
        }
      }
    }
  }
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 1);
    sum[i] += __shfl_xor_sync(0xffffffffu, sum[i], 2);
    const int r = warp * 16 + (lane >> 2) + 8 * i;
    if (r >= rows) continue;
    const float f = 1.f / sum[i];
    const bf16* g = a.gate + (size_t)(row0 + r) * a.ldp + h * a.dv;
    bf16* dst = a.out + (size_t)(row0 + r) * a.n_out + h * a.dv;
#pragma unroll
    for (int nd = 0; nd < DV / 8; ++nd) {
      if (nd < nv) {
        const int d = nd * 8 + (lane & 3) * 2;
        const float2 gg = bf162_bits_to_f2(*reinterpret_cast<const uint32_t*>(g + d));
        *reinterpret_cast<uint32_t*>(dst + d) = f2_to_bf162_bits(o[nd][2 * i] * f * sigmoid_f(gg.x), o[nd][2 * i + 1] * f * sigmoid_f(gg.y));
      }
    }
  }
  if (h == 0)
    for (int x = tid; x < rows * (a.n_out - a.heads * a.dv); x += 256) {
      const int w = a.n_out - a.heads * a.dv;
      a.out[(size_t)(row0 + x / w) * a.n_out + a.heads * a.dv + x % w] = __float2bfloat16(0.f);
    }
}

template <int CW> cudaError_t decode_launch(DecArgs a, int tiles, int B, cudaStream_t st) {
  const size_t q_bytes = (size_t)(16 * (a.kch * 16 + 16) + 127) / 128 * 128, stage = (size_t)TILE * a.kch * 16;
  int stages = 4;
  while (stages > 2 && q_bytes + stages * stage > 100 * 1024) --stages;          // two blocks on an SM where three stages allow it
  if (stages < 3 && q_bytes + 3 * stage <= (size_t)LD_SMEM) stages = 3;
  const size_t smem = q_bytes + stages * stage + 128;
  if (smem > (size_t)LD_SMEM + 128) return cudaErrorInvalidValue;
  a.n_stages = stages;
  auto k = latent_decode_kernel<CW>;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, LD_SMEM + 128);
    if (e != cudaSuccess) return e;
    cudaFuncSetAttribute(k, cudaFuncAttributePreferredSharedMemoryCarveout, 100);
    configured = true;
  }
  return trl_launch(k, dim3(tiles * a.n_splits, B), dim3(288), smem, st, a);
}

template <int DQ, int DV> cudaError_t prompt_launch(const PromptArgs& a, cudaStream_t st) {
  constexpr int smem = 128 * DQ * 2 + 2 * TILE * (DQ + DV) * 2 + 128;
  auto k = latent_prompt_kernel<DQ, DV>;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return e;
    configured = true;
  }
  return trl_launch(k, dim3((a.n + 127) / 128, a.heads), dim3(256), smem, st, a);
}

}  // namespace

// 1 when the tensor-core forms take heads of these (padded) sizes.
TRL_API int trl_latent_mma_ok(int dk, int rd, int dv, int kv) {
  const size_t row = (size_t)(kv + rd) * 2;
  return dk + rd <= 256 && dv <= 256 && kv <= 512 && 16 * (row + 16) + 128 + 2 * TILE * row <= (size_t)LD_SMEM;
}

// Sequences of min_len..max_len tokens in the absorbed form.  q: [T, heads, dq], whose rotated part is turned here (n_pairs 0: it
// already is); ukt: [heads][kv][dk]; uv: [heads * dv, kv]; ql: [T, heads, kv + rd]; part: fp32 [T, heads, n_splits, kv]; ml:
// [T, heads, n_splits] pairs; tiles: 16-row tiles of the longest sequence; gate: gate columns of the fused projection rows.
TRL_API int trl_latent_decode(const void* q, int dq, int dk, int rd, const void* ukt, const void* uv, int kv, int dv, const void* freqs,
                              int n_pairs, float amp, void* ql, const void* pages, int n_blocks, const void* table, int max_blocks,
                              const void* q_start, const void* q_len, const void* positions, const void* seq_ids, void* part, void* ml,
                              const void* gate, int ldp, void* out, int n_out, int T, int B, int tiles, int heads, int n_splits, int window,
                              int min_len, int max_len, float scale, void* stream) {
  if (T <= 0 || B <= 0 || tiles <= 0 || heads <= 0 || dk % 16 || rd % 16 || dv % 16 || kv % 16 || dk + rd != dq || n_splits < 1 ||
      n_splits > MAX_SPLITS || window < 1 || n_blocks <= 0 || n_out < heads * dv || 2 * n_pairs > rd || !trl_latent_mma_ok(dk, rd, dv, kv) ||
      ((uintptr_t)pages & 15) || ((uintptr_t)q & 15) || ((uintptr_t)ukt & 15) || ((uintptr_t)uv & 15))
    return (int)cudaErrorInvalidValue;
  cudaStream_t st = (cudaStream_t)stream;
  const int groups = (T + 7) / 8;
  cudaError_t e = trl_launch(latent_absorb_kernel, dim3(heads, (kv + 127) / 128, groups), dim3(256), (size_t)8 * (dk + 8) * sizeof(bf16), st,
                             (const bf16*)q, dq, dk, rd, (const bf16*)ukt, kv, (const double*)freqs, n_pairs, amp, (const int*)positions,
                             (const int*)seq_ids, (const int*)q_len, max_len, (bf16*)ql, T, heads);
  if (e != cudaSuccess) return (int)e;
  DecArgs a;
  a.ql = (const bf16*)ql, a.pages = (const unsigned char*)pages, a.kch = (kv + rd) / 8, a.vch = kv / 8, a.n_blocks = n_blocks;
  a.table = (const int*)table, a.max_blocks = max_blocks, a.q_start = (const int*)q_start, a.q_len = (const int*)q_len;
  a.positions = (const int*)positions, a.part = (float*)part, a.ml = (float2*)ml, a.heads = heads, a.n_splits = n_splits, a.n_stages = 2;
  a.window = window, a.min_len = min_len, a.max_len = max_len, a.scale2 = scale * LOG2E;
  if (kv <= 128) e = decode_launch<16>(a, tiles, B, st);
  else if (kv <= 256) e = decode_launch<32>(a, tiles, B, st);
  else e = decode_launch<64>(a, tiles, B, st);
  if (e != cudaSuccess) return (int)e;
  const int z = groups * heads >= 148 ? 1 : (dv > 128 ? 2 : 1);
  return (int)trl_launch(latent_out_kernel, dim3(heads, groups, z), dim3(256), (size_t)2 * 8 * (kv + 8) * sizeof(bf16), st, (const float*)part,
                         (const float2*)ml, n_splits, (const bf16*)uv, kv, dv, (const bf16*)gate, ldp, (bf16*)out, n_out, (const int*)seq_ids,
                         (const int*)q_start, (const int*)q_len, (const int*)positions, T, heads, window, max_len);
}

// Cached rows of positions lo .. lo + n - 1 of one sequence (table: its row of the block table).
TRL_API int trl_latent_gather(const void* pages, int n_blocks, const void* table, int lo, int n, int kv, int rd, void* c, void* kr, void* stream) {
  if (n <= 0 || lo < 0 || kv % 16 || rd % 16 || n_blocks <= 0) return (int)cudaErrorInvalidValue;
  return (int)trl_launch(latent_gather_kernel, dim3(n), dim3(64), 0, (cudaStream_t)stream, (const unsigned char*)pages, n_blocks,
                         (const int*)table, lo, (kv + rd) / 8, kv / 8, (bf16*)c, (bf16*)kr);
}

// One sequence's n query tokens (pointers at its first token) against expanded keys of positions lo .. lo + n_keys - 1.
TRL_API int trl_latent_prompt(const void* q, int dq, int dk, int rd, int dv, const void* kvx, int ldkv, const void* kr, const void* gate, int ldp,
                              void* out, int n_out, const void* positions, int n, int lo, int n_keys, int heads, int window, float scale,
                              void* stream) {
  if (n <= 0 || n_keys <= 0 || heads <= 0 || dk % 16 || rd % 16 || dv % 16 || dk + rd != dq || dq > 256 || dv > 256 || ldkv % 8 || ldp % 2 ||
      ldkv < heads * (dk + dv) || n_out < heads * dv || window < 1 || ((uintptr_t)q & 15) || ((uintptr_t)kvx & 15) || ((uintptr_t)kr & 15))
    return (int)cudaErrorInvalidValue;
  PromptArgs a;
  a.q = (const bf16*)q, a.kvx = (const bf16*)kvx, a.kr = (const bf16*)kr, a.gate = (const bf16*)gate, a.out = (bf16*)out;
  a.positions = (const int*)positions, a.n = n, a.lo = lo, a.n_keys = n_keys, a.heads = heads, a.dq = dq, a.dk = dk, a.rd = rd, a.dv = dv;
  a.ldkv = ldkv, a.ldp = ldp, a.n_out = n_out, a.window = window, a.scale2 = scale * LOG2E;
  cudaStream_t st = (cudaStream_t)stream;
  if (dv <= 128 && dq <= 128) return (int)prompt_launch<128, 128>(a, st);
  if (dv <= 128 && dq <= 192) return (int)prompt_launch<192, 128>(a, st);
  return (int)prompt_launch<256, 256>(a, st);
}
