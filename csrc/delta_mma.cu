// Delta rule with one decay per key channel for prompts (forms: delta.cu): 32 tokens at a time.  With G_i the running sum of a chunk's log
// decays per channel, and S_0 the state before it, the rule unrolls to
//
//   A_ij = beta_i sum_d k_i k_j e^(G_i - G_j) (j < i),  N_ij = sum_d q_i k_j e^(G_i - G_j) (j <= i),  T = (1 + A)^-1
//   u = T (beta v) - T (beta k e^G) S_0,   o = (q e^G) S_0 + N u,   S = e^(G_C) S_0 + (k e^(G_C - G))^T u
//
// so that what depends on q, k, v and decays alone is formed for all chunks at once, and only four small products are left on the way from
// state to state.  No exponent is above zero.
//
//   delta_form_kernel   a block per (chunk, head, sequence): A, N, T, W = T (beta k e^G), U = T (beta v) and the decayed q and k, in
//                       fp32; goes out as one record whose tiles have the order in which the scan's shared memory wants them.
//   delta_scan_kernel   a block per (head, 32 or 64 value columns, sequence), four warps on mma.sync: chunk after chunk, the state in fp32
//                       registers.  Every operand enters its products as a bf16 pair (value and rest; three products), so it keeps 16
//                       bits of mantissa; sums are fp32.  Each half of a record is copied (cp.async) while the other half is used.
// Reference parity: the reference's chunked delta rule has one decay per head (no counterpart).
#include "delta.cuh"

// The sequences and chunks of a launch (mirrored by tilerl_b200/ops/cuda_gated.py::DeltaSel).
struct DeltaSel {
  int n, c0, nc, pad;                  // sequences; chunks c0 .. c0 + nc - 1 of each
  int seq[64];
};

namespace {

constexpr int DC = 32;                                          // tokens of a chunk
constexpr int DF_THREADS = 288, DS_THREADS = 128;
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ float ex2_f(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
// byte offset of 16-byte chunk c of row r
template <int ROW> __device__ __forceinline__ uint32_t tile_off(int r, int c) {
  if constexpr (ROW >= 128) return (uint32_t)(r * ROW + ((c ^ (r & 7)) << 4));
  else return (uint32_t)(r * ROW + ((c ^ ((r >> 1) & 3)) << 4));
}

// A record: bf16 pairs (value, rest) of W, q e^G and k e^(G_C - G) [32, DK] and of N [32, 32], then e^(G_C) [DK], then U by slices of 32 columns.
template <int DK> struct Rec {
  static constexpr int ROW = DK * 2, TILE = DC * ROW, NROW = DC * 2, NTILE = DC * NROW, USLICE = DC * 32 * 4;
  static constexpr int N = 6 * TILE, G = N + 2 * NTILE, U = G + DK * 4;
  static __host__ __device__ size_t bytes(int dv) { return (size_t)U + (size_t)(dv + 31) / 32 * USLICE; }
};

template <int DK> struct FormSmem {
  static constexpr int LD = DK + 4;
  float q[DC][LD], k[DC][LD], g[DC][LD], G[DC][LD];              // g: factors, G: running sums (powers of two)
  float A[DC][DC + 1];
  __align__(16) float T[DC][DC + 4];
  float beta[DC];
};

template <int DK>
__global__ void __launch_bounds__(DF_THREADS) delta_form_kernel(const DeltaArgs a, const DeltaSel sel) {
  using R = Rec<DK>;
  using SM = FormSmem<DK>;
  constexpr int Q4 = DK / 4;
  extern __shared__ __align__(16) unsigned char df_raw[];
  SM& sm = *reinterpret_cast<SM*>(df_raw);
  pdl_launch_dependents(72);
  pdl_wait();
  const int h = blockIdx.y, seq = sel.seq[blockIdx.z], i0 = (sel.c0 + (int)blockIdx.x) * DC, T_ = a.q_len[seq];
  if (i0 >= T_) return;
  const int n = min(DC, T_ - i0), kh = h / (a.heads / a.kv_heads), tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const size_t t0 = (size_t)a.q_start[seq] + i0;
  unsigned char* rec = reinterpret_cast<unsigned char*>(a.chunk) + (((size_t)blockIdx.z * sel.nc + blockIdx.x) * a.heads + h) * R::bytes(a.dv);
  for (int x = tid; x < DC * Q4; x += DF_THREADS) {              // rows past the sequence and columns past the head: zeros
    const int r = x / Q4, d = x % Q4 * 4;
    float4 q = make_float4(0.f, 0.f, 0.f, 0.f), k = q, l = q;
    if (r < n && d < a.dk) {
      q = load4(a.q + ((t0 + r) * a.kv_heads + kh) * a.dk + d), k = load4(a.k + ((t0 + r) * a.kv_heads + kh) * a.dk + d);
      l = load4(a.keep + ((t0 + r) * a.heads + h) * a.dk + d);
    }
    *reinterpret_cast<float4*>(&sm.q[r][d]) = q, *reinterpret_cast<float4*>(&sm.k[r][d]) = k;
    *reinterpret_cast<float4*>(&sm.G[r][d]) = make_float4(l.x * LOG2E, l.y * LOG2E, l.z * LOG2E, l.w * LOG2E);
  }
  if (tid < DC) sm.beta[tid] = tid < n ? a.beta[(t0 + tid) * a.heads + h] : 0.f;
  __syncthreads();
  if (tid < DK) {
    float s = 0.f;
#pragma unroll 8
    for (int r = 0; r < DC; ++r) {
      const float l = sm.G[r][tid];
      s += l;
      sm.g[r][tid] = ex2_f(l), sm.G[r][tid] = s;
    }
    reinterpret_cast<float*>(rec + R::G)[tid] = ex2_f(s);
  }
  __syncthreads();
  // ---- A and N in tiles of four by four, eight threads (shares of the channels) a tile
  {
    const int tile = tid >> 3, sl = tid & 7;
    int ti = 0;
    while ((ti + 1) * (ti + 2) / 2 <= tile) ++ti;
    const int tj = tile - ti * (ti + 1) / 2, r = 4 * ti, c = 4 * tj;
    const bool diag = ti == tj;
    float acc[32];                                               // k . k, then q . k, row by row
#pragma unroll
    for (int i = 0; i < 32; ++i) acc[i] = 0.f;
#pragma unroll 1
    for (int s = 0; s < DK / 16; ++s) {
      const int d = (8 * s + sl) * 2;
      auto get = [&](const float* p) { return *reinterpret_cast<const float2*>(p); };
      float2 kr[4], qr[4], kc[4], gr[4], gc[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) kr[i] = get(&sm.k[r + i][d]), qr[i] = get(&sm.q[r + i][d]), kc[i] = get(&sm.k[c + i][d]);
#pragma unroll
      for (int i = 1; i < 4; ++i) gr[i] = get(&sm.g[r + i][d]), gc[i] = get(&sm.g[c + i][d]);
      const float2 Gr = get(&sm.G[r][d]), Gc = get(&sm.G[c + 3][d]);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        auto at = [&](const float2& v) { return e ? v.y : v.x; };
        // e^(G_i - G_j): the closest pair of rows, the others by factors (on the diagonal: one, and factors below it)
        float E[4];
        E[3] = diag ? 0.f : ex2_f(at(Gr) - at(Gc));
        E[2] = E[3] * at(gc[3]), E[1] = E[2] * at(gc[2]), E[0] = diag ? 1.f : E[1] * at(gc[1]);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          if (i) {
#pragma unroll
            for (int j = 0; j < 4; ++j) E[j] = diag && j == i ? 1.f : E[j] * at(gr[i]);
          }
#pragma unroll
          for (int j = 0; j < 4; ++j) {
            const float x = at(kc[j]) * E[j];
            acc[i * 4 + j] = fmaf(at(kr[i]), x, acc[i * 4 + j]), acc[16 + i * 4 + j] = fmaf(at(qr[i]), x, acc[16 + i * 4 + j]);
          }
        }
      }
    }
    // the eight shares: every step halves what a thread holds, until it has one row of one product
#pragma unroll
    for (int m = 4, n = 16; m > 0; m >>= 1, n >>= 1)
#pragma unroll
      for (int i = 0; i < n; ++i) {
        const float mine = sl & m ? acc[n + i] : acc[i], other = sl & m ? acc[i] : acc[n + i];
        acc[i] = mine + __shfl_xor_sync(0xffffffffu, other, m);
      }
    const int row = r + (sl & 3);
    if (sl < 4) {
#pragma unroll
      for (int j = 0; j < 4; ++j) sm.A[row][c + j] = c + j < row ? sm.beta[row] * acc[j] : 0.f;
    } else {
      uint2 hi, lo;                                              // (zeros above the diagonal)
      split2(acc[0], acc[1], hi.x, lo.x), split2(acc[2], acc[3], hi.y, lo.y);
      const uint32_t o = tile_off<R::NROW>(row, c >> 3) + (c & 7) * 2;
      *reinterpret_cast<uint2*>(rec + R::N + o) = hi, *reinterpret_cast<uint2*>(rec + R::N + R::NTILE + o) = lo;
      if (!diag) {                                               // the mirrored tile lies above the diagonal
        const uint32_t m = tile_off<R::NROW>(c + (sl & 3), r >> 3) + (r & 7) * 2;
        *reinterpret_cast<uint2*>(rec + R::N + m) = make_uint2(0u, 0u), *reinterpret_cast<uint2*>(rec + R::N + R::NTILE + m) = make_uint2(0u, 0u);
      }
    }
  }
  __syncthreads();
  if (warp == 0) {
    // ---- the two diagonal blocks of T: a lane solves a column of its block by forward substitution
    const int o = lane & 16, j = lane & 15;
    float t[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      float v0 = i == j ? 1.f : 0.f, v1 = 0.f;
#pragma unroll
      for (int m = 0; m < i; ++m) {
        if (m & 1) v1 = fmaf(-sm.A[o + i][o + m], t[m], v1);
        else v0 = fmaf(-sm.A[o + i][o + m], t[m], v0);
      }
      t[i] = v0 + v1;
      sm.T[o + i][lane] = t[i];
      if (o) sm.T[i][lane] = 0.f;
    }
  } else {
    // ---- decayed queries and keys
    for (int x = tid - 32; x < 2 * DC * (DK / 8); x += DF_THREADS - 32) {
      const bool is_k = x >= DC * (DK / 8);
      const int y = is_k ? x - DC * (DK / 8) : x, r = y / (DK / 8), ch = y % (DK / 8);
      uint32_t hi[4], lo[4];
#pragma unroll
      for (int e = 0; e < 4; e += 2) {
        const int d = ch * 8 + 2 * e;
        const float4 f = *reinterpret_cast<const float4*>(is_k ? &sm.k[r][d] : &sm.q[r][d]);
        float4 g = *reinterpret_cast<const float4*>(&sm.G[r][d]);
        if (is_k) {
          const float4 end = *reinterpret_cast<const float4*>(&sm.G[DC - 1][d]);
          g = make_float4(end.x - g.x, end.y - g.y, end.z - g.z, end.w - g.w);
        }
        split2(f.x * ex2_f(g.x), f.y * ex2_f(g.y), hi[e], lo[e]);
        split2(f.z * ex2_f(g.z), f.w * ex2_f(g.w), hi[e + 1], lo[e + 1]);
      }
      unsigned char* dst = rec + (is_k ? 4 : 2) * R::TILE + tile_off<R::ROW>(r, ch);
      *reinterpret_cast<uint4*>(dst) = make_uint4(hi[0], hi[1], hi[2], hi[3]);
      *reinterpret_cast<uint4*>(dst + R::TILE) = make_uint4(lo[0], lo[1], lo[2], lo[3]);
    }
  }
  __syncthreads();
  // ---- the block below: -T22 (A21 T11), the inner product where A is not needed any more
  if (tid < 256) {
    const int i = tid >> 4, j = tid & 15;
    float v = 0.f;
#pragma unroll
    for (int m = 0; m < 16; ++m) v = fmaf(sm.A[16 + i][m], sm.T[m][j], v);
    sm.A[i][j] = v;
  }
  __syncthreads();
  if (tid < 256) {
    const int i = tid >> 4, j = tid & 15;
    float v = 0.f;
#pragma unroll
    for (int m = 0; m < 16; ++m) v = fmaf(-sm.T[16 + i][16 + m], sm.A[m][j], v);
    sm.T[16 + i][j] = v;
  }
  __syncthreads();
  // ---- W and U: a thread per column (pairs of lanes store W together)
  const int cols = DK + (a.dv + 31) / 32 * 32;
  for (int x0 = 0; x0 < cols; x0 += DF_THREADS) {
    const int x = x0 + tid;
    const bool is_w = x < DK, in = x < cols;
    float y[DC];
    if (is_w) {
#pragma unroll
      for (int r = 0; r < DC; ++r) y[r] = sm.beta[r] * sm.k[r][x] * ex2_f(sm.G[r][x]);
    } else {
      const bf16* v = reinterpret_cast<const bf16*>(a.v) + (t0 * a.heads + h) * a.dv + (x - DK);
#pragma unroll
      for (int r = 0; r < DC; ++r) y[r] = in && r < n && x - DK < a.dv ? sm.beta[r] * __bfloat162float(v[(size_t)r * a.heads * a.dv]) : 0.f;
    }
#pragma unroll
    for (int i = 0; i < DC; ++i) {
      float s0 = 0.f, s1 = 0.f;
#pragma unroll
      for (int j = 0; j <= i; j += 4) {
        const float4 t = *reinterpret_cast<const float4*>(&sm.T[i][j]);      // (zeros above the diagonal)
        s0 = fmaf(t.x, y[j], s0), s1 = fmaf(t.y, y[j + 1], s1), s0 = fmaf(t.z, y[j + 2], s0), s1 = fmaf(t.w, y[j + 3], s1);
      }
      const float s = s0 + s1, other = __shfl_xor_sync(0xffffffffu, s, 1);
      if (is_w) {
        const bool odd = x & 1;
        uint32_t hi, lo;
        split2(odd ? other : s, odd ? s : other, hi, lo);
        *reinterpret_cast<uint32_t*>(rec + (odd ? R::TILE : 0) + tile_off<R::ROW>(i, x >> 3) + (x & 6) * 2) = odd ? lo : hi;
      } else if (in) {
        const int c = x - DK;
        reinterpret_cast<float*>(rec + R::U + (c >> 5) * R::USLICE)[i * 32 + (c & 31)] = s;
      }
    }
  }
}

template <int DK, int DV> struct ScanSm {
  static constexpr int HEAD = Rec<DK>::U, VROW = DV * 2;
  __align__(128) unsigned char st[HEAD], u[DV / 32 * Rec<DK>::USLICE];
  __align__(128) unsigned char s_hi[DK * VROW], s_lo[DK * VROW], d_hi[DC * VROW], d_lo[DC * VROW];
};

template <int DK, int DV>
__global__ void __launch_bounds__(DS_THREADS, 2) delta_scan_kernel(const DeltaArgs a, const DeltaSel sel) {
  using R = Rec<DK>;
  using SM = ScanSm<DK, DV>;
  constexpr int MT = DK / 64, NT = DV / 8, NH = NT / 2, VROW = SM::VROW;
  extern __shared__ __align__(128) unsigned char ds_raw[];
  SM& sm = *reinterpret_cast<SM*>(ds_raw);
  pdl_launch_dependents(73);
  pdl_wait();
  const int n_sl = (a.dv + DV - 1) / DV, h = blockIdx.x / n_sl, slice = blockIdx.x % n_sl, col0 = slice * DV, seq = sel.seq[blockIdx.y];
  const int T_ = a.q_len[seq], first = sel.c0, last = min(sel.c0 + sel.nc, (T_ + DC - 1) / DC);
  if (first >= last) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, t4 = lane & 3;
  const size_t t0 = a.q_start[seq];
  const int slot = a.slots[seq];
  float* s_rec = a.states + (size_t)slot * a.slot_stride + (size_t)a.cur[slot] * a.plane_stride + (size_t)h * a.dk * a.dv + col0;
  auto u32 = [](const void* p) { return (uint32_t)__cvta_generic_to_shared(p); };
  const uint32_t base = u32(sm.st), u_a = u32(sm.u), sh_a = u32(sm.s_hi), sl_a = u32(sm.s_lo), dh_a = u32(sm.d_hi), dl_a = u32(sm.d_lo);
  const size_t rec_bytes = R::bytes(a.dv);
  const unsigned char* recs = reinterpret_cast<const unsigned char*>(a.chunk) + ((size_t)blockIdx.y * sel.nc * a.heads + h) * rec_bytes;
  const int u_bytes = min(DV / 32, (a.dv + 31) / 32 - slice * (DV / 32)) * R::USLICE;
  // a record comes in two parts: what the products with the state need (W, q, U), then what those with u need (k, N, factors)
  auto stage1 = [&](int c) {
    const unsigned char* src = recs + (size_t)(c - sel.c0) * a.heads * rec_bytes;
#pragma unroll 8
    for (int x = tid * 16; x < 4 * R::TILE; x += DS_THREADS * 16) cp16(base + x, src + x);
    for (int x = tid * 16; x < u_bytes; x += DS_THREADS * 16) cp16(u_a + x, src + R::U + slice * (DV / 32) * R::USLICE + x);
    cp_commit();
  };
  auto stage2 = [&](int c) {
    const unsigned char* src = recs + (size_t)(c - sel.c0) * a.heads * rec_bytes;
#pragma unroll 8
    for (int x = 4 * R::TILE + tid * 16; x < SM::HEAD; x += DS_THREADS * 16) cp16(base + x, src + x);
    cp_commit();
  };
  stage1(first);

  // rows of the state this warp owns: 16 (MT warp + mt) .. + 15
  float S[MT][NT][4];
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int r = (MT * warp + mt) * 16 + g8 + 8 * i, c = nt * 8 + 2 * t4;
        float2 v = make_float2(0.f, 0.f);
        if (r < a.dk && col0 + c < a.dv) v = *reinterpret_cast<const float2*>(s_rec + (size_t)r * a.dv + c);
        S[mt][nt][2 * i] = v.x, S[mt][nt][2 * i + 1] = v.y;
      }
  auto publish = [&]() {                    // the state as the B operand of W S and q S
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          uint32_t hi, lo;
          split2(S[mt][nt][2 * i], S[mt][nt][2 * i + 1], hi, lo);
          const uint32_t o = tile_off<VROW>((MT * warp + mt) * 16 + g8 + 8 * i, nt) + t4 * 4;
          *reinterpret_cast<uint32_t*>(sm.s_hi + o) = hi, *reinterpret_cast<uint32_t*>(sm.s_lo + o) = lo;
        }
  };
  publish();
  const int lrow = (lane & 7) + ((lane >> 3) & 1) * 8, lch = lane >> 4;      // rows / chunk of A and transposed B tiles
  const int brow = (lane & 7) + (lane >> 4) * 8, bch = (lane >> 3) & 1;      // of transposed A tiles
  const int mrow = 16 * (warp & 1), n0 = (warp >> 1) * NH;                   // this warp's tokens and columns (in eights)
  for (int c = first; c < last; ++c) {
    cp_wait<0>();
    __syncthreads();                        // the first part and the state's copy are in; the second part's place is free
    stage2(c);
    // ---- P = W S, O = q S of this warp's 16 tokens and columns; main products and rests in sums of their own
    float P[NH][4], O[NH][4], X[NH][4], Y[NH][4];
#pragma unroll
    for (int nt = 0; nt < NH; ++nt)
#pragma unroll
      for (int e = 0; e < 4; ++e) P[nt][e] = O[nt][e] = X[nt][e] = Y[nt][e] = 0.f;
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk) {
      uint32_t wh[4], wl[4], qh[4], ql[4];
      const uint32_t o = base + tile_off<R::ROW>(mrow + lrow, kk * 2 + lch);
      ldsm4(wh, o), ldsm4(wl, o + R::TILE), ldsm4(qh, o + 2 * R::TILE), ldsm4(ql, o + 3 * R::TILE);
#pragma unroll
      for (int nt = 0; nt < NH; nt += 2) {
        uint32_t sh[4], sl[4];
        const uint32_t so = tile_off<VROW>(kk * 16 + lrow, n0 + nt + lch);
        ldsm4t(sh, sh_a + so), ldsm4t(sl, sl_a + so);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          mma16(P[nt + i], wh, sh[2 * i], sh[2 * i + 1]);
          mma16(O[nt + i], qh, sh[2 * i], sh[2 * i + 1]);
          mma16(X[nt + i], wl, sh[2 * i], sh[2 * i + 1]);
          mma16(Y[nt + i], ql, sh[2 * i], sh[2 * i + 1]);
          mma16(X[nt + i], wh, sl[2 * i], sl[2 * i + 1]);
          mma16(Y[nt + i], qh, sl[2 * i], sl[2 * i + 1]);
        }
      }
    }
    // ---- u = U - P, kept as the B operand of the next two products
#pragma unroll
    for (int nt = 0; nt < NH; ++nt)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int r = mrow + g8 + 8 * i, cc = (n0 + nt) * 8 + 2 * t4;
        float2 u = make_float2(0.f, 0.f);
        if (col0 + cc < a.dv) u = *reinterpret_cast<const float2*>(sm.u + (cc >> 5) * R::USLICE + (r * 32 + (cc & 31)) * 4);
        uint32_t hi, lo;
        split2(u.x - (P[nt][2 * i] + X[nt][2 * i]), u.y - (P[nt][2 * i + 1] + X[nt][2 * i + 1]), hi, lo);
        const uint32_t o = tile_off<VROW>(r, n0 + nt) + t4 * 4;
        *reinterpret_cast<uint32_t*>(sm.d_hi + o) = hi, *reinterpret_cast<uint32_t*>(sm.d_lo + o) = lo;
      }
    cp_wait<0>();
    __syncthreads();                        // u and the second part are in; the first part's place is free
    if (c + 1 < last) stage1(c + 1);
    // ---- O += N u
#pragma unroll
    for (int kt = 0; kt < DC / 16; ++kt) {
      if (kt <= (warp & 1)) {
        uint32_t nh[4], nl[4];
        const uint32_t o = base + R::N + tile_off<R::NROW>(mrow + lrow, kt * 2 + lch);
        ldsm4(nh, o), ldsm4(nl, o + R::NTILE);
#pragma unroll
        for (int nt = 0; nt < NH; nt += 2) {
          uint32_t dh[4], dl[4];
          const uint32_t dd = tile_off<VROW>(16 * kt + lrow, n0 + nt + lch);
          ldsm4t(dh, dh_a + dd), ldsm4t(dl, dl_a + dd);
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            mma16(O[nt + i], nh, dh[2 * i], dh[2 * i + 1]);
            mma16(Y[nt + i], nl, dh[2 * i], dh[2 * i + 1]);
            mma16(Y[nt + i], nh, dl[2 * i], dl[2 * i + 1]);
          }
        }
      }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int t = c * DC + mrow + g8 + 8 * i;
      if (t < T_) {
        float* dst = a.o + ((t0 + t) * a.heads + h) * a.dv + col0;
#pragma unroll
        for (int nt = 0; nt < NH; ++nt) {
          const int cc = (n0 + nt) * 8 + 2 * t4;
          if (col0 + cc < a.dv) *reinterpret_cast<float2*>(dst + cc) = make_float2(O[nt][2 * i] + Y[nt][2 * i], O[nt][2 * i + 1] + Y[nt][2 * i + 1]);
        }
      }
    }
    // ---- S = e^(G_C) S + (decayed keys)^T u
    const float* eg = reinterpret_cast<const float*>(sm.st + R::G);
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      const float f0 = eg[(MT * warp + mt) * 16 + g8], f1 = eg[(MT * warp + mt) * 16 + g8 + 8];
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) S[mt][nt][0] *= f0, S[mt][nt][1] *= f0, S[mt][nt][2] *= f1, S[mt][nt][3] *= f1;
    }
#pragma unroll
    for (int kt = 0; kt < DC / 16; ++kt) {
      uint32_t kh[MT][4], kl[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        const uint32_t o = base + 4 * R::TILE + tile_off<R::ROW>(16 * kt + brow, (MT * warp + mt) * 2 + bch);
        ldsm4t(kh[mt], o), ldsm4t(kl[mt], o + R::TILE);
      }
#pragma unroll
      for (int nt = 0; nt < NT; nt += 2) {
        uint32_t dh[4], dl[4];
        const uint32_t dd = tile_off<VROW>(16 * kt + lrow, nt + lch);
        ldsm4t(dh, dh_a + dd), ldsm4t(dl, dl_a + dd);
#pragma unroll
        for (int mt = 0; mt < MT; ++mt)
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            mma16(S[mt][nt + i], kh[mt], dh[2 * i], dh[2 * i + 1]);
            mma16(S[mt][nt + i], kl[mt], dh[2 * i], dh[2 * i + 1]);
            mma16(S[mt][nt + i], kh[mt], dl[2 * i], dl[2 * i + 1]);
          }
      }
    }
    publish();                              // (the old copy's last readers are behind the barrier above)
  }
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int nt = 0; nt < NT; ++nt)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int r = (MT * warp + mt) * 16 + g8 + 8 * i, c = nt * 8 + 2 * t4;
        if (r < a.dk && col0 + c < a.dv)
          *reinterpret_cast<float2*>(s_rec + (size_t)r * a.dv + c) = make_float2(S[mt][nt][2 * i], S[mt][nt][2 * i + 1]);
      }
}

template <int DK, int DV> cudaError_t scan_launch(const DeltaArgs& a, const DeltaSel& s, cudaStream_t st) {
  auto k = delta_scan_kernel<DK, DV>;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(ScanSm<DK, DV>));
    if (e != cudaSuccess) return e;
    cudaFuncSetAttribute(k, cudaFuncAttributePreferredSharedMemoryCarveout, 100);
    configured = true;
  }
  return trl_launch(k, dim3(a.heads * ((a.dv + DV - 1) / DV), s.n), dim3(DS_THREADS), sizeof(ScanSm<DK, DV>), st, a, s);
}
template <int DK> cudaError_t chunk_launch(const DeltaArgs& a, const DeltaSel& s, int narrow, cudaStream_t st) {
  auto k = delta_form_kernel<DK>;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(FormSmem<DK>));
    if (e != cudaSuccess) return e;
    cudaFuncSetAttribute(k, cudaFuncAttributePreferredSharedMemoryCarveout, 100);
    configured = true;
  }
  const cudaError_t e = trl_launch(k, dim3(s.nc, a.heads, s.n), dim3(DF_THREADS), sizeof(FormSmem<DK>), st, a, s);
  if (e != cudaSuccess) return e;
  return narrow ? scan_launch<DK, 32>(a, s, st) : scan_launch<DK, 64>(a, s, st);
}

}  // namespace

// Bytes of one chunk of one head in the scratch of trl_delta_chunk.
TRL_API int trl_delta_record(int dk, int dv) { return (int)(dk <= 64 ? Rec<64>::bytes(dv) : Rec<128>::bytes(dv)); }
// Tokens of a chunk.
TRL_API int trl_delta_chunk_tokens() { return DC; }

// bf16 values, dk up to 128, no kept states: chunks c0 .. c0 + nc - 1 of the selected sequences, whose rows trl_delta_prep has prepared.
// a.chunk: n * nc * heads records.  narrow: 32 value columns a block instead of 64 (more blocks).
TRL_API int trl_delta_chunk(const DeltaArgs* args, const DeltaSel* sel, int narrow, void* stream) {
  const DeltaArgs& a = *args;
  if (delta_args_bad(a) || a.dk > 128 || a.keep_flags || !a.states || !a.o || !a.cur || !a.q_start || !a.q_len || !a.slots || !a.chunk ||
      ((uintptr_t)a.chunk & 15) || sel->n < 1 || sel->n > 64 || sel->nc < 1 || sel->c0 < 0 || a.slot_stride % 2 || a.plane_stride % 2 ||
      ((uintptr_t)a.states & 7) || ((uintptr_t)a.o & 7) || ((uintptr_t)a.q & 15) || ((uintptr_t)a.k & 15) || ((uintptr_t)a.keep & 15))
    return (int)cudaErrorInvalidValue;
  return (int)(a.dk <= 64 ? chunk_launch<64>(a, *sel, narrow, (cudaStream_t)stream) : chunk_launch<128>(a, *sel, narrow, (cudaStream_t)stream));
}
