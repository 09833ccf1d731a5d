// Decayed scans of prompts on tensor cores (mma.sync bf16): 64 tokens at a time, chunk after chunk (forms: scan.cu).
//
// Within a chunk every weight is one exponential of a difference: with L the running sum of the log decays, r_s the log
// of what token s adds minus L_s, and M_t the running maximum of r and of the old state's m (mLSTM; -L_t for the others, whose
// maximum is not tracked),
//
//   o_t = exp(m_0 - M_t) S_0^T q_t + sum_{s <= t} exp(r_s - M_t) b_s (q_t . k_s) v_s
//   S   = exp(m_0 - M_C) S_0      + sum_s        exp(r_s - M_C) b_s  k_s v_s^T          m = L_C + M_C
//
// One block = (head, 32 or 64 value columns, sequence), four warps; a warp owns 16 tokens of the chunk as rows of the score
// tile and dk / 4 rows of the state, which stays in fp32 registers from chunk to chunk.  q, k and v are bf16 as projected;
// scores, weights, decayed keys and the state enter their products as bf16 pairs (value and rest), so they keep 16 bits
// of mantissa and the sums are fp32.  The next chunk's rows are copied (cp.async) while this one is computed.
// Reference parity: the reference's chunked recurrence is Gated DeltaNet (no counterpart).
#include "scan.cuh"

namespace {

constexpr int SC = 64, SM_THREADS = 128;

template <int DK, int DV> struct ScanSmem {
  static constexpr int KROW = DK * 2, VROW = DV * 2;
  __align__(128) unsigned char q[2][SC * KROW], k[2][SC * KROW], v[2][SC * VROW];
  __align__(128) unsigned char s_hi[DK * VROW], s_lo[DK * VROW];
  float r[SC], m[SC], b[SC], c[SC], keep[SC], floor_[SC], nq[SC], n[DK];
  float last;                               // exp(m_0 - M_C)
};

// byte offset of 16-byte chunk c of row r
template <int ROW> __device__ __forceinline__ uint32_t sm_off(int r, int c) {
  if constexpr (ROW >= 128) return (uint32_t)(r * ROW + ((c ^ (r & 7)) << 4));
  else return (uint32_t)(r * ROW + ((c ^ ((r >> 1) & 3)) << 4));
}
__device__ __forceinline__ void cp16z(uint32_t dst, const void* src, bool in) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(in ? 16 : 0) : "memory");
}

template <int KIND, int DK, int DV>
__global__ void __launch_bounds__(SM_THREADS) scan_chunk_kernel(const ScanArgs a) {
  using SM = ScanSmem<DK, DV>;
  constexpr int KROW = SM::KROW, VROW = SM::VROW, MT = DK / 64, NT = DV / 8;
  extern __shared__ __align__(128) unsigned char sm_raw[];
  SM& sm = *reinterpret_cast<SM*>(sm_raw);
  pdl_launch_dependents(43);
  pdl_wait();
  const int n_sl = (a.dv + DV - 1) / DV, h = blockIdx.x / n_sl, slice = blockIdx.x % n_sl, col0 = slice * DV, seq = blockIdx.y;
  const int T_ = a.q_len[seq], t0 = a.q_start[seq];
  if (T_ < a.min_len || T_ > a.max_len) return;
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g8 = lane >> 2, t4 = lane & 3;
  const int slot = a.slots[seq];
  float* rec = a.states + (size_t)slot * a.slot_stride + (size_t)a.cur[slot] * a.plane_stride;
  const int copies = (a.dv + 31) / 32, copy0 = h * copies + slice * (DV / 32), n_copy = min(DV / 32, copies - slice * (DV / 32));
  float* n_rec = rec + (size_t)a.heads * a.dk * a.dv;
  float* m_rec = n_rec + (size_t)a.heads * copies * a.dk;
  float* s_rec = rec + (size_t)h * a.dk * a.dv + col0;
  auto u32 = [](const void* p) { return (uint32_t)__cvta_generic_to_shared(p); };
  const uint32_t q_a[2] = {u32(sm.q[0]), u32(sm.q[1])}, k_a[2] = {u32(sm.k[0]), u32(sm.k[1])}, v_a[2] = {u32(sm.v[0]), u32(sm.v[1])};
  const uint32_t hi_a = u32(sm.s_hi), lo_a = u32(sm.s_lo);

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
  auto publish = [&]() {                    // the state as the B operand of q . S
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          uint32_t hi, lo;
          split2(S[mt][nt][2 * i], S[mt][nt][2 * i + 1], hi, lo);
          const uint32_t o = sm_off<VROW>((MT * warp + mt) * 16 + g8 + 8 * i, nt) + t4 * 4;
          *reinterpret_cast<uint32_t*>(sm.s_hi + o) = hi;
          *reinterpret_cast<uint32_t*>(sm.s_lo + o) = lo;
        }
  };
  publish();
  float m_run = 0.f;                        // the state's running maximum (warp 0)
  if (KIND == SCAN_MLSTM) {
    for (int d = tid; d < DK; d += SM_THREADS) sm.n[d] = d < a.dk ? n_rec[(size_t)copy0 * a.dk + d] : 0.f;
    m_run = m_rec[copy0];
  }
  const bf16* base = reinterpret_cast<const bf16*>(a.rows) + (size_t)t0 * a.ld;
  const int qc = a.q0 + (h / a.per) * a.dk, kc = a.k0 + (h / a.per) * a.dk, vc = a.v0 + h * a.dv + col0;
  auto stage = [&](int i0, int b) {         // rows past the sequence and columns past the head come as zeros
#pragma unroll
    for (int x = tid; x < SC * (DK / 8); x += SM_THREADS) {
      const int r = x / (DK / 8), c = x % (DK / 8);
      const bool in = i0 + r < T_ && c * 8 < a.dk;
      const bf16* row = base + (size_t)(in ? i0 + r : 0) * a.ld + (in ? c * 8 : 0);
      cp16z(q_a[b] + sm_off<KROW>(r, c), row + qc, in);
      cp16z(k_a[b] + sm_off<KROW>(r, c), row + kc, in);
    }
#pragma unroll
    for (int x = tid; x < SC * (DV / 8); x += SM_THREADS) {
      const int r = x / (DV / 8), c = x % (DV / 8);
      const bool in = i0 + r < T_ && col0 + c * 8 < a.dv;
      cp16z(v_a[b] + sm_off<VROW>(r, c), base + (size_t)(in ? i0 + r : 0) * a.ld + (in ? vc + c * 8 : 0), in);
    }
    cp_commit();
  };
  float g0[2], g1[2];                       // raw gates of this lane's two tokens of the next chunk (warp 0)
  auto fetch_gates = [&](int i0) {
    if (warp != 0) return;
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int j = i0 + 2 * lane + e;
      g0[e] = g1[e] = 0.f;
      if (KIND != SCAN_FIXED && j < T_) {
        const float* row = a.gates + (size_t)(t0 + j) * a.ldg;
        g0[e] = row[h];
        if (KIND == SCAN_MLSTM) g1[e] = row[a.heads + h];
      }
    }
  };
  const float bias0 = KIND != SCAN_FIXED ? a.gate_b[h] : 0.f, bias1 = KIND == SCAN_MLSTM ? a.gate_b[a.heads + h] : 0.f;
  const float rate = KIND == SCAN_MAMBA2 ? expf(a.a_log[h]) : KIND == SCAN_FIXED ? a.a_log[h] : 0.f, skip = KIND == SCAN_MAMBA2 ? a.skip[h] : 0.f;
  fetch_gates(0);
  stage(0, 0);
  const int lrow = (lane & 7) + ((lane >> 3) & 1) * 8, lch = lane >> 4;      // rows / chunk of A and transposed B tiles
  const int brow = (lane & 7) + (lane >> 4) * 8, bch = (lane >> 3) & 1;      // of B tiles stored [n][k]; also of transposed A tiles
  int b = 0;
  for (int i0 = 0; i0 < T_; i0 += SC, b ^= 1) {
    const int nb = min(SC, T_ - i0);
    cp_wait<0>();
    __syncthreads();                        // this chunk's rows and the state copy are in; the other buffer is free
    if (i0 + SC < T_) stage(i0 + SC, b ^ 1);
    if (warp == 0) {
      // ---- the chunk's scalars: lane owns tokens 2 lane and 2 lane + 1
      float la[2], add[2], bb[2];
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const bool in = 2 * lane + e < nb;
        if (KIND == SCAN_MAMBA2) {
          bb[e] = in ? softplus_x(g0[e] + bias0) : 0.f;
          la[e] = -rate * bb[e], add[e] = 0.f;
        } else if (KIND == SCAN_FIXED) {
          bb[e] = in ? 1.f : 0.f, la[e] = in ? rate : 0.f, add[e] = 0.f;
        } else {
          add[e] = in ? a.cap * tanhf((g0[e] + bias0) / a.cap) : -INFINITY;
          la[e] = in ? -softplus_x(-a.cap * tanhf((g1[e] + bias1) / a.cap)) : 0.f;
          bb[e] = 1.f;
        }
      }
      float sum = la[0] + la[1];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float up = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= o) sum += up;
      }
      const float L[2] = {sum - la[1], sum};
      const float r[2] = {add[0] - L[0], add[1] - L[1]};
      float M[2];
      if (KIND == SCAN_MLSTM) {
        float mx = fmaxf(r[0], r[1]);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
          const float up = __shfl_up_sync(0xffffffffu, mx, o);
          if (lane >= o) mx = fmaxf(mx, up);
        }
        float before = __shfl_up_sync(0xffffffffu, mx, 1);
        before = lane == 0 ? m_run : fmaxf(before, m_run);
        M[0] = fmaxf(before, r[0]), M[1] = fmaxf(M[0], r[1]);
      } else {
        M[0] = -L[0], M[1] = -L[1];
      }
      const float M_end = __shfl_sync(0xffffffffu, M[1], 31), L_end = __shfl_sync(0xffffffffu, L[1], 31);
#pragma unroll
      for (int e = 0; e < 2; ++e) {
        const int j = 2 * lane + e;
        sm.r[j] = r[e], sm.m[j] = M[e], sm.b[j] = bb[e];
        sm.c[j] = expf(r[e] - M_end) * bb[e];
        sm.keep[j] = expf(m_run - M[e]);
        if (KIND == SCAN_MLSTM) sm.floor_[j] = expf(-(L[e] + M[e]));
      }
      if (lane == 0) sm.last = expf(m_run - M_end);
      if (KIND == SCAN_MLSTM) m_run = L_end + M_end;
    }
    if (i0 + SC < T_) fetch_gates(i0 + SC);
    // ---- q . k of this warp's 16 tokens against tokens up to its own, and q . S
    float sc[4][2][4], O[NT][4];
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int n8 = 0; n8 < 2; ++n8) sc[j][n8][0] = sc[j][n8][1] = sc[j][n8][2] = sc[j][n8][3] = 0.f;
#pragma unroll
    for (int nt = 0; nt < NT; ++nt) O[nt][0] = O[nt][1] = O[nt][2] = O[nt][3] = 0.f;
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk) {
      uint32_t qf[4];
      ldsm4(qf, q_a[b] + sm_off<KROW>(16 * warp + lrow, kk * 2 + lch));
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        if (j <= warp) {
          uint32_t kf[4];
          ldsm4(kf, k_a[b] + sm_off<KROW>(16 * j + brow, kk * 2 + bch));
          mma16(sc[j][0], qf, kf[0], kf[1]);
          mma16(sc[j][1], qf, kf[2], kf[3]);
        }
      }
#pragma unroll
      for (int nt = 0; nt < NT; nt += 2) {
        uint32_t f[4];
        ldsm4t(f, hi_a + sm_off<VROW>(kk * 16 + lrow, nt + lch));
        mma16(O[nt], qf, f[0], f[1]);
        mma16(O[nt + 1], qf, f[2], f[3]);
        ldsm4t(f, lo_a + sm_off<VROW>(kk * 16 + lrow, nt + lch));
        mma16(O[nt], qf, f[0], f[1]);
        mma16(O[nt + 1], qf, f[2], f[3]);
      }
    }
    if (KIND == SCAN_MLSTM) {               // q . n: two threads per token
      const int r = tid >> 1, half = tid & 1;
      float d = 0.f;
#pragma unroll
      for (int c = 0; c < DK / 16; ++c) {
        const int ch = half * (DK / 16) + c;
        float f[8];
        Chunk<bf16>::get(*reinterpret_cast<const uint4*>(sm.q[b] + sm_off<KROW>(r, ch)), f);
#pragma unroll
        for (int e = 0; e < 8; ++e) d = fmaf(f[e], sm.n[ch * 8 + e], d);
      }
      d += __shfl_xor_sync(0xffffffffu, d, 1);
      if (half == 0) sm.nq[r] = d;
    }
    __syncthreads();                        // scalars and q . n are in; the state copy and n have been read
    // ---- weights; O = keep (q . S) + W v
    const float M0 = sm.m[16 * warp + g8], M1 = sm.m[16 * warp + g8 + 8];
    {
      const float k0 = sm.keep[16 * warp + g8], k1 = sm.keep[16 * warp + g8 + 8];
#pragma unroll
      for (int nt = 0; nt < NT; ++nt) O[nt][0] *= k0, O[nt][1] *= k0, O[nt][2] *= k1, O[nt][3] *= k1;
    }
    float row[2] = {0.f, 0.f};
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      if (j <= warp) {
        uint32_t wh[4], wl[4];
#pragma unroll
        for (int n8 = 0; n8 < 2; ++n8) {
          const int s = 16 * j + 8 * n8 + 2 * t4;
          const float2 r = *reinterpret_cast<const float2*>(&sm.r[s]), bb = *reinterpret_cast<const float2*>(&sm.b[s]);
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const float M = i ? M1 : M0;
            const int t = 16 * warp + g8 + 8 * i;
            const float w0 = s <= t ? sc[j][n8][2 * i] * __expf(r.x - M) * bb.x : 0.f;
            const float w1 = s + 1 <= t ? sc[j][n8][2 * i + 1] * __expf(r.y - M) * bb.y : 0.f;
            row[i] += w0 + w1;
            split2(w0, w1, wh[n8 * 2 + i], wl[n8 * 2 + i]);
          }
        }
#pragma unroll
        for (int nt = 0; nt < NT; nt += 2) {
          uint32_t f[4];
          ldsm4t(f, v_a[b] + sm_off<VROW>(16 * j + lrow, nt + lch));
          mma16(O[nt], wh, f[0], f[1]);
          mma16(O[nt + 1], wh, f[2], f[3]);
          mma16(O[nt], wl, f[0], f[1]);
          mma16(O[nt + 1], wl, f[2], f[3]);
        }
      }
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int t = 16 * warp + g8 + 8 * i;
      float f = 1.f;
      if (KIND == SCAN_MLSTM) {
        float d = row[i];
        d += __shfl_xor_sync(0xffffffffu, d, 1);
        d += __shfl_xor_sync(0xffffffffu, d, 2);
        d = fmaf(sm.keep[t], sm.nq[t], d) * a.q_scale;
        f = a.q_scale / (fmaxf(fabsf(d), sm.floor_[t]) + 1e-6f);
      }
      if (t < nb) {
        float* dst = a.o + ((size_t)(t0 + i0 + t) * a.heads + h) * a.dv + col0;
#pragma unroll
        for (int nt = 0; nt < NT; ++nt) {
          const int c = nt * 8 + 2 * t4;
          if (col0 + c < a.dv) {
            float2 y = make_float2(O[nt][2 * i] * f, O[nt][2 * i + 1] * f);
            if (KIND == SCAN_MAMBA2) {
              const float2 x = bf162_bits_to_f2(*reinterpret_cast<const uint32_t*>(sm.v[b] + sm_off<VROW>(t, nt) + t4 * 4));
              y.x = fmaf(skip, x.x, y.x), y.y = fmaf(skip, x.y, y.y);
            }
            *reinterpret_cast<float2*>(dst + c) = y;
          }
        }
      }
    }
    // ---- S = last S + (decayed keys)^T v
    const float last = sm.last;
#pragma unroll
    for (int mt = 0; mt < MT; ++mt)
#pragma unroll
      for (int nt = 0; nt < NT; ++nt)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[mt][nt][e] *= last;
#pragma unroll
    for (int kt = 0; kt < SC / 16; ++kt) {
      const float2 c0 = *reinterpret_cast<const float2*>(&sm.c[16 * kt + 2 * t4]);
      const float2 c1 = *reinterpret_cast<const float2*>(&sm.c[16 * kt + 8 + 2 * t4]);
      uint32_t kh[MT][4], kl[MT][4];
#pragma unroll
      for (int mt = 0; mt < MT; ++mt) {
        uint32_t kf[4];
        ldsm4t(kf, k_a[b] + sm_off<KROW>(16 * kt + brow, (MT * warp + mt) * 2 + bch));
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const float2 f = bf162_bits_to_f2(kf[e]), c = e < 2 ? c0 : c1;
          split2(f.x * c.x, f.y * c.y, kh[mt][e], kl[mt][e]);
        }
      }
#pragma unroll
      for (int nt = 0; nt < NT; nt += 2) {
        uint32_t f[4];
        ldsm4t(f, v_a[b] + sm_off<VROW>(16 * kt + lrow, nt + lch));
#pragma unroll
        for (int mt = 0; mt < MT; ++mt) {
          mma16(S[mt][nt], kh[mt], f[0], f[1]);
          mma16(S[mt][nt + 1], kh[mt], f[2], f[3]);
          mma16(S[mt][nt], kl[mt], f[0], f[1]);
          mma16(S[mt][nt + 1], kl[mt], f[2], f[3]);
        }
      }
    }
    if (KIND == SCAN_MLSTM && tid < DK) {
      float n = sm.n[tid] * last;
      for (int s = 0; s < SC; ++s)
        n = fmaf(__bfloat162float(*reinterpret_cast<const bf16*>(sm.k[b] + sm_off<KROW>(s, tid >> 3) + (tid & 7) * 2)), sm.c[s], n);
      sm.n[tid] = n;
    }
    publish();
  }
  __syncthreads();
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
  if (KIND == SCAN_MLSTM)
    for (int cp = 0; cp < n_copy; ++cp) {
      for (int d = tid; d < a.dk; d += SM_THREADS) n_rec[(size_t)(copy0 + cp) * a.dk + d] = sm.n[d];
      if (tid == 0) m_rec[copy0 + cp] = m_run;
    }
}

template <int KIND, int DK, int DV> cudaError_t chunk_launch(const ScanArgs& a, int B, cudaStream_t st) {
  auto k = scan_chunk_kernel<KIND, DK, DV>;
  static bool configured = false;
  if (!configured) {
    const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(ScanSmem<DK, DV>));
    if (e != cudaSuccess) return e;
    configured = true;
  }
  return trl_launch(k, dim3(a.heads * ((a.dv + DV - 1) / DV), B), dim3(SM_THREADS), sizeof(ScanSmem<DK, DV>), st, a);
}
template <int KIND> cudaError_t chunk_any(const ScanArgs& a, int B, int narrow, cudaStream_t st) {
  if (a.dk <= 64) return narrow ? chunk_launch<KIND, 64, 32>(a, B, st) : chunk_launch<KIND, 64, 64>(a, B, st);
  return narrow ? chunk_launch<KIND, 128, 32>(a, B, st) : chunk_launch<KIND, 128, 64>(a, B, st);
}

}  // namespace

// bf16 rows, dk up to 128, no kept states.  narrow: 32 value columns a block instead of 64 (more blocks, scores formed
// twice as often).  Serves sequences of min_len..max_len tokens.
TRL_API int trl_scan_chunk(const ScanArgs* a, int B, int kind, int narrow, void* stream) {
  if (B <= 0 || scan_args_bad(*a, kind) || a->dk > 128 || a->keep_flags || a->ld % 8 || a->q0 % 8 || a->k0 % 8 || a->v0 % 8 ||
      a->slot_stride % 2 || a->plane_stride % 2 || ((uintptr_t)a->rows & 15) || ((uintptr_t)a->states & 7))
    return (int)cudaErrorInvalidValue;
  cudaStream_t st = (cudaStream_t)stream;
  if (kind == SCAN_FIXED) return (int)chunk_any<SCAN_FIXED>(*a, B, narrow, st);
  return (int)(kind == SCAN_MAMBA2 ? chunk_any<SCAN_MAMBA2>(*a, B, narrow, st) : chunk_any<SCAN_MLSTM>(*a, B, narrow, st));
}
