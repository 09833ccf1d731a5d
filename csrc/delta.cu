// Delta rule with one decay per key channel (models/tobadra.py).  Per head, with g_t the factors the rows of S keep:
//
//   S <- g_t S;   u = beta_t (v_t - S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t
//
//   delta_prep_kernel    a tick's rows, a block per token: causal convolution and silu (earlier rows from the slot's ring), unit length of
//                        every q / k head, log g = -exp(A) softplus(low + bias) per channel, beta = sigmoid(gate).
//   delta_serial_kernel  token after token, 32 value columns of a head per block, the state in registers: decoding, windows of kept
//                        states, short portions, and fp32 models.  o = (g S)^T q + (k . q) u, so a token needs one block barrier.
//   delta_step_kernel    one token per sequence from projection rows to normed and gated ones (heads up to 128 x 128).
//   (prompts: delta_mma.cu; the norm and gate behind it: scan_norm_kernel of scan.cu)
//
// q, k, decays, beta, state and sums are fp32; v is in the compute type, as its convolution leaves it.
// Reference parity: the reference's delta rule has one decay per head (kernels_gdn.py of tilerl-kernels; no counterpart).
#include "delta.cuh"

namespace {

// silu of a short convolution
template <typename T> __device__ __forceinline__ float conv_silu(float x) {
  return sizeof(T) == 2 ? __fdividef(x, 1.f + __expf(-x)) : x * sigmoid_x(x);
}

template <typename T>
__global__ void __launch_bounds__(512, 2) delta_prep_kernel(const DeltaArgs a) {
  constexpr int C = Chunk<T>::N;
  extern __shared__ __align__(16) float s_row[];               // [2 k0] convolved q and k
  pdl_launch_dependents(70);
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nt = blockDim.x, nw = nt >> 5;
  const int pos = a.positions[t], seq = a.seq_ids[t], t0 = a.q_start[seq];
  const T* row = reinterpret_cast<const T*>(a.rows) + (size_t)t * a.ldp;
  T* ring = reinterpret_cast<T*>(a.ring) + (size_t)a.slots[seq] * a.ring_slot;
  for (int c = tid * C; c < a.channels; c += nt * C) {
    const uint4 own = *reinterpret_cast<const uint4*>(row + c);
    float f[C], acc[C];
#pragma unroll
    for (int e = 0; e < C; ++e) acc[e] = 0.f;
#pragma unroll 4
    for (int back = 0; back < a.taps; ++back) {
      if (back > pos) break;
      const T* src = t - back >= t0 ? row - (size_t)back * a.ldp + c : ring + (size_t)((pos - back) % a.ring_rows) * a.ring_ld + c;
      Chunk<T>::get(*reinterpret_cast<const uint4*>(src), f);
#pragma unroll
      for (int e = 0; e < C; e += 4) {
        const float4 w = __ldg(reinterpret_cast<const float4*>(a.conv_w + (size_t)(a.taps - 1 - back) * a.channels + c + e));
        acc[e] = fmaf(f[e], w.x, acc[e]), acc[e + 1] = fmaf(f[e + 1], w.y, acc[e + 1]);
        acc[e + 2] = fmaf(f[e + 2], w.z, acc[e + 2]), acc[e + 3] = fmaf(f[e + 3], w.w, acc[e + 3]);
      }
    }
#pragma unroll
    for (int e = 0; e < C; ++e) acc[e] = conv_silu<T>(acc[e]);
    if (a.write_ring) *reinterpret_cast<uint4*>(ring + (size_t)(pos % a.ring_rows) * a.ring_ld + c) = own;
    const uint4 out = Chunk<T>::put(acc);
    if (c >= a.v0) {
      *reinterpret_cast<uint4*>(reinterpret_cast<T*>(a.v) + (size_t)t * a.heads * a.dv + c - a.v0) = out;
    } else {
      Chunk<T>::get(out, f);                                   // (as the compute type holds it)
#pragma unroll
      for (int e = 0; e < C; e += 4) *reinterpret_cast<float4*>(s_row + c + e) = make_float4(f[e], f[e + 1], f[e + 2], f[e + 3]);
    }
  }
  const int n = a.heads * a.dk;
  for (int c = tid * 4; c < n; c += nt * 4) {
    const float4 x = load4(a.low + (size_t)t * n + c), b = __ldg(reinterpret_cast<const float4*>(a.dt_bias + c));
    const float r = -expf(a.a_log[c / a.dk]);
    *reinterpret_cast<float4*>(a.keep + (size_t)t * n + c) =
        make_float4(r * softplus_x(x.x + b.x), r * softplus_x(x.y + b.y), r * softplus_x(x.z + b.z), r * softplus_x(x.w + b.w));
  }
  for (int h = tid; h < a.heads; h += nt) a.beta[(size_t)t * a.heads + h] = sigmoid_x(a.gates[(size_t)t * a.ldg + h]);
  __syncthreads();
  for (int h = warp; h < 2 * a.kv_heads; h += nw) {
    const float* src = s_row + h * a.dk;
    float ss = 0.f;
    for (int d = lane; d < a.dk; d += 32) ss = fmaf(src[d], src[d], ss);
    const bool is_q = h < a.kv_heads;
    const float f = (is_q ? a.q_scale : 1.f) / sqrtf(warp_sum(ss) + 1e-6f);
    float* dst = (is_q ? a.q : a.k) + ((size_t)t * a.kv_heads + (is_q ? h : h - a.kv_heads)) * a.dk;
    for (int d = lane; d < a.dk; d += 32) dst[d] = src[d] * f;
  }
}

// grid (heads * column slices, sequences), 256 threads: lane = column, warp = dk / 8 state rows
template <typename T, int RMAX>
__global__ void __launch_bounds__(256, RMAX <= 16 ? 4 : 2) delta_serial_kernel(const DeltaArgs a) {
  constexpr int DK = RMAX * 8, TB = RMAX <= 16 ? 16 : 8;
  __shared__ float s_q[TB][DK], s_k[TB][DK], s_g[TB][DK], s_v[TB][32], s_beta[TB], s_kq[TB];
  __shared__ float s_p[2][8][32], s_o[2][8][32];
  pdl_launch_dependents(71);
  const int n_sl = (a.dv + 31) / 32, h = blockIdx.x / n_sl, col0 = (blockIdx.x % n_sl) * 32, seq = blockIdx.y, kh = h / (a.heads / a.kv_heads);
  const int T_ = a.q_len[seq], t0 = a.q_start[seq];
  if (T_ < a.min_len || T_ > a.max_len) {
    pdl_wait();                              // (a launch ends no sooner than those before it)
    return;
  }
  const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, R = a.dk / 8, col = col0 + lane;
  const int slot = a.slots[seq], plane = a.cur[slot];
  const bool keep_all = a.keep_flags && a.keep_flags[seq];
  float* rec = a.states + (size_t)slot * a.slot_stride;
  const size_t s_off = ((size_t)h * a.dk + warp * R) * a.dv + col;
  float S[RMAX];
  {
    // (before the dependency wait: the state's last writer is the previous tick, and every tick has launches in between that let their
    // dependents in only after their own wait)
    const float* src = rec + (size_t)plane * a.plane_stride;
#pragma unroll
    for (int r = 0; r < RMAX; ++r) S[r] = r < R && col < a.dv ? src[s_off + (size_t)r * a.dv] : 0.f;
  }
  pdl_wait();
  auto save = [&](int pl) {
    float* dst = rec + (size_t)pl * a.plane_stride;
#pragma unroll
    for (int r = 0; r < RMAX; ++r)
      if (r < R && col < a.dv) dst[s_off + (size_t)r * a.dv] = S[r];
  };
  const T* vb = reinterpret_cast<const T*>(a.v);
  for (int i0 = 0; i0 < T_; i0 += TB) {
    const int nb = min(TB, T_ - i0);
    __syncthreads();
    for (int x = tid; x < nb * a.dk; x += 256) {
      const int j = x / a.dk, d = x % a.dk;
      const size_t t = t0 + i0 + j;
      s_q[j][d] = a.q[(t * a.kv_heads + kh) * a.dk + d];
      s_k[j][d] = a.k[(t * a.kv_heads + kh) * a.dk + d];
      s_g[j][d] = expf(a.keep[(t * a.heads + h) * a.dk + d]);
    }
    for (int x = tid; x < nb * 32; x += 256)
      s_v[x >> 5][x & 31] = col0 + (x & 31) < a.dv ? to_f(vb[((size_t)(t0 + i0 + (x >> 5)) * a.heads + h) * a.dv + col0 + (x & 31)]) : 0.f;
    if (tid < nb) s_beta[tid] = a.beta[(size_t)(t0 + i0 + tid) * a.heads + h];
    __syncthreads();
    for (int j = warp; j < nb; j += 8) {
      float d = 0.f;
      for (int c = lane; c < a.dk; c += 32) d = fmaf(s_q[j][c], s_k[j][c], d);
      d = warp_sum(d);
      if (lane == 0) s_kq[j] = d;
    }
    __syncthreads();
    for (int j = 0; j < nb; ++j) {
      const float *kr = &s_k[j][warp * R], *qr = &s_q[j][warp * R], *gr = &s_g[j][warp * R];
      float p = 0.f, o = 0.f;
#pragma unroll
      for (int r = 0; r < RMAX; ++r) {
        if (r < R) {
          S[r] *= gr[r];
          p = fmaf(kr[r], S[r], p);
          o = fmaf(qr[r], S[r], o);
        }
      }
      s_p[j & 1][warp][lane] = p, s_o[j & 1][warp][lane] = o;
      __syncthreads();
      p = 0.f;
#pragma unroll
      for (int w = 0; w < 8; ++w) p += s_p[j & 1][w][lane];
      const float u = s_beta[j] * (s_v[j][lane] - p);
#pragma unroll
      for (int r = 0; r < RMAX; ++r)
        if (r < R) S[r] = fmaf(kr[r], u, S[r]);
      if (keep_all) save(i0 + j);
      if (warp == 0 && col < a.dv) {
        o = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) o += s_o[j & 1][w][lane];
        a.o[((size_t)(t0 + i0 + j) * a.heads + h) * a.dv + col] = fmaf(s_kq[j], u, o);
      }
    }
  }
  if (!keep_all) save(plane);
}

// One token per sequence, preparation and norm included: grid (heads, sequences); a warp owns 32 columns and a quarter of the rows.
constexpr int DT_COLS = 128;
template <typename T, int RMAX>
__global__ void __launch_bounds__(512, 2) delta_step_kernel(const DeltaArgs a, const T* gate, int ldg, const float* __restrict__ norm, T* out, int ldo,
                                                         int vdim, float eps) {
  __shared__ float s_q[4 * RMAX], s_k[4 * RMAX], s_g[4 * RMAX], s_v[DT_COLS], s_p[4][DT_COLS], s_o[4][DT_COLS], s_sum[3], s_ss[4];
  pdl_launch_dependents(74);
  const int h = blockIdx.x, seq = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nt = blockDim.x;
  if (a.q_len[seq] == 0) {
    pdl_wait();
    return;
  }
  const int grp = warp & 3, col = (warp >> 2) * 32 + lane, R = a.dk / 4, t = a.q_start[seq], slot = a.slots[seq];
  const bool in = col < a.dv;
  float* st = a.states + (size_t)slot * a.slot_stride + (size_t)a.cur[slot] * a.plane_stride + ((size_t)h * a.dk + grp * R) * a.dv + col;
  float S[RMAX];
#pragma unroll
  for (int r = 0; r < RMAX; ++r) S[r] = r < R && in ? st[(size_t)r * a.dv] : 0.f;      // (before the wait: see delta_serial_kernel)
  pdl_wait();
  const int per = a.heads / a.kv_heads, kh = h / per, pos = a.positions[t];
  const T* row = reinterpret_cast<const T*>(a.rows) + (size_t)t * a.ldp;
  T* ring = reinterpret_cast<T*>(a.ring) + (size_t)slot * a.ring_slot;
  for (int x = tid; x < 2 * a.dk + a.dv; x += nt) {
    const bool is_v = x >= 2 * a.dk, is_k = !is_v && x >= a.dk;
    const int c = is_v ? a.v0 + h * a.dv + x - 2 * a.dk : is_k ? a.k0 + kh * a.dk + x - a.dk : kh * a.dk + x;
    const T own = row[c];
    float v = 0.f;
#pragma unroll 4
    for (int j = 0; j < a.taps; ++j) {
      const int back = a.taps - 1 - j;
      if (back <= pos) v = fmaf(to_f(back ? ring[(size_t)((pos - back) % a.ring_rows) * a.ring_ld + c] : own), a.conv_w[(size_t)j * a.channels + c], v);
    }
    v = to_f(from_f<T>(conv_silu<T>(v)));
    if (is_v) s_v[x - 2 * a.dk] = v;
    else if (is_k) s_k[x - a.dk] = v;
    else s_q[x] = v;
    if (is_v || h % per == 0) ring[(size_t)(pos % a.ring_rows) * a.ring_ld + c] = own;      // (no block reads this row of the ring)
  }
  const float rate = -expf(a.a_log[h]);
  for (int d = tid; d < a.dk; d += nt) s_g[d] = expf(rate * softplus_x(a.low[((size_t)t * a.heads + h) * a.dk + d] + a.dt_bias[h * a.dk + d]));
  __syncthreads();
  if (warp < 3) {                              // q . q, k . k, q . k
    const float *x = warp == 1 ? s_k : s_q, *y = warp == 0 ? s_q : s_k;
    float d = 0.f;
    for (int c = lane; c < a.dk; c += 32) d = fmaf(x[c], y[c], d);
    d = warp_sum(d);
    if (lane == 0) s_sum[warp] = d;
  }
  float p = 0.f, o = 0.f;
#pragma unroll
  for (int r = 0; r < RMAX; ++r)
    if (r < R) {
      S[r] *= s_g[grp * R + r];
      p = fmaf(s_k[grp * R + r], S[r], p), o = fmaf(s_q[grp * R + r], S[r], o);
    }
  s_p[grp][col] = p, s_o[grp][col] = o;
  __syncthreads();
  const float fq = a.q_scale / sqrtf(s_sum[0] + 1e-6f), fk = 1.f / sqrtf(s_sum[1] + 1e-6f);
  p = (s_p[0][col] + s_p[1][col] + s_p[2][col] + s_p[3][col]) * fk;
  const float beta = sigmoid_x(a.gates[(size_t)t * a.ldg + h]), u = in ? beta * (s_v[col] - p) : 0.f;
#pragma unroll
  for (int r = 0; r < RMAX; ++r)
    if (r < R && in) st[(size_t)r * a.dv] = fmaf(s_k[grp * R + r] * fk, u, S[r]);
  float y = 0.f;
  if (grp == 0) {
    if (in) y = fmaf(s_sum[2] * fq * fk, u, (s_o[0][col] + s_o[1][col] + s_o[2][col] + s_o[3][col]) * fq);
    const float ss = warp_sum(y * y);          // (padding columns hold zeros)
    if (lane == 0) s_ss[warp >> 2] = ss;
  }
  __syncthreads();
  if (grp == 0) {
    float ss = 0.f;
    for (int w = 0; w * 32 < a.dv; ++w) ss += s_ss[w];
    const int c = h * a.dv + col;
    if (in) out[(size_t)t * ldo + c] = from_f<T>(y * inv_rms(ss, vdim, eps) * norm[c] * sigmoid_x(to_f(gate[(size_t)t * ldg + c])));
  }
  if (h == 0)
    for (int c = a.heads * a.dv + tid; c < ldo; c += nt) out[(size_t)t * ldo + c] = from_f<T>(0.f);
}

template <typename T> cudaError_t serial_launch(const DeltaArgs& a, int B, cudaStream_t st) {
  const dim3 grid(a.heads * ((a.dv + 31) / 32), B);
  if (a.dk <= 32) return trl_launch(delta_serial_kernel<T, 4>, grid, dim3(256), 0, st, a);
  if (a.dk <= 64) return trl_launch(delta_serial_kernel<T, 8>, grid, dim3(256), 0, st, a);
  if (a.dk <= 128) return trl_launch(delta_serial_kernel<T, 16>, grid, dim3(256), 0, st, a);
  return trl_launch(delta_serial_kernel<T, 32>, grid, dim3(256), 0, st, a);
}

}  // namespace

// args: filled by the caller.  write_ring: the rows go into the ring (one token per sequence; else trl_ring_store does it afterwards).
TRL_API int trl_delta_prep(const DeltaArgs* args, int T, int f32, void* stream) {
  const DeltaArgs& a = *args;
  const int per = f32 ? 4 : 8;
  const size_t smem = (size_t)2 * a.k0 * sizeof(float);
  if (T <= 0 || delta_args_bad(a) || smem > 200 * 1024 || a.taps < 1 || a.taps > a.ring_rows || a.ldp % per || a.channels > a.ldp || a.ldg < a.heads ||
      a.ring_ld % per || a.ring_slot % per || !a.rows || !a.conv_w || !a.ring || !a.low || !a.dt_bias || !a.a_log || !a.gates || !a.positions ||
      !a.seq_ids || !a.q_start || !a.slots || ((uintptr_t)a.rows & 15) || ((uintptr_t)a.ring & 15) || ((uintptr_t)a.low & 15) || ((uintptr_t)a.keep & 15))
    return (int)cudaErrorInvalidValue;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(delta_prep_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_prep_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const int threads = T <= 148 && a.channels >= 4096 ? 512 : 256;
  if (f32) return (int)trl_launch(delta_prep_kernel<float>, dim3(T), dim3(threads), smem, (cudaStream_t)stream, a);
  return (int)trl_launch(delta_prep_kernel<bf16>, dim3(T), dim3(threads), smem, (cudaStream_t)stream, a);
}

// Serves sequences of min_len..max_len tokens, whose rows trl_delta_prep has prepared.
TRL_API int trl_delta_serial(const DeltaArgs* args, int B, int f32, void* stream) {
  const DeltaArgs& a = *args;
  if (B <= 0 || delta_args_bad(a) || !a.states || !a.o || !a.cur || !a.q_start || !a.q_len || !a.slots) return (int)cudaErrorInvalidValue;
  return (int)(f32 ? serial_launch<float>(a, B, (cudaStream_t)stream) : serial_launch<bf16>(a, B, (cudaStream_t)stream));
}

// Heads that trl_delta_step takes.
TRL_API int trl_delta_step_ok(int dk, int dv) { return dk <= 128 && dv <= DT_COLS; }

// One token per sequence, no kept states: rows -> out [T, ldo], normed per head (over vdim values), times norm [heads * dv], times
// sigmoid(gate [T, ldg]); the state moves on and the rows go into the ring.  a.q, a.k, a.v, a.keep, a.beta and a.o are not used.
TRL_API int trl_delta_step(const DeltaArgs* args, int B, const void* gate, int ldg, const void* norm, void* out, int ldo, int vdim, float eps,
                           int f32, void* stream) {
  const DeltaArgs& a = *args;
  if (B <= 0 || a.heads <= 0 || a.kv_heads <= 0 || a.heads % a.kv_heads || a.dk <= 0 || a.dk % 16 || a.dv <= 0 || a.dv % 16 || !trl_delta_step_ok(a.dk, a.dv) ||
      a.keep_flags || !a.states || !a.cur || !a.q_start || !a.q_len || !a.slots || !a.positions || !a.rows || !a.conv_w || !a.ring || !a.low || !a.dt_bias ||
      !a.a_log || !a.gates || a.taps < 1 || a.taps > a.ring_rows || a.ldg < a.heads || !gate || !norm || !out || ldo < a.heads * a.dv ||
      ldg < a.heads * a.dv || vdim < 1 || vdim > a.dv || a.k0 != a.kv_heads * a.dk || a.v0 != 2 * a.k0 || a.channels != a.v0 + a.heads * a.dv)
    return (int)cudaErrorInvalidValue;
  const dim3 grid(a.heads, B), block((a.dv + 31) / 32 * 128);
  cudaStream_t st = (cudaStream_t)stream;
#define DELTA_STEP(TT, RR)                                                                                                             \
  return (int)trl_launch(delta_step_kernel<TT, RR>, grid, block, 0, st, a, (const TT*)gate, ldg, (const float*)norm, (TT*)out, ldo, vdim, eps)
  if (f32) {
    if (a.dk <= 64) DELTA_STEP(float, 16);
    DELTA_STEP(float, 32);
  }
  if (a.dk <= 64) DELTA_STEP(bf16, 16);
  DELTA_STEP(bf16, 32);
#undef DELTA_STEP
}
