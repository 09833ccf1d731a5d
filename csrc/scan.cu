// Decayed scans: S_t = keep_t S_(t-1) + add_t k_t v_t^T, o_t = S_t^T q_t per head, in three forms (models/fetotar.py, models/tobadra.py).
//
//   Mamba-2   keep = exp(-exp(A) dt), add = dt, dt = softplus(raw + bias); k = B, q = C of the head's group and v = x, all
//             after a causal convolution and silu; o += D x; then o silu(z), RMS norm in groups, weight.
//   mLSTM     log gates i = cap tanh(raw / cap), f = logsigmoid(cap tanh(raw / cap)) and a running maximum m:
//             m_t = max(f + m_(t-1), i), keep = exp(f + m_(t-1) - m_t), add = exp(i - m_t); beside S the sum n of the keys,
//             and o is divided by max(|n . q|, exp(-m)) + 1e-6; then RMS norm per head, weight, sigmoid gate.
//
//   fixed     keep = a constant of the head, add = 1; RMS norm over all heads, weight, sigmoid gate.
//
//   scan_conv_kernel    convolution of a tick's rows (with or without silu, inputs with or without a bias, with or without the input itself added); rows before the tick's
//                       first token come from the slot's ring.
//   conv_run_kernel     the same for prompts (up to 4 taps).
//   ring_store_kernel   a tick's last convolution inputs into the ring.
//   scan_serial_kernel  token after token, 32 value columns of a head per block, the state in registers: decoding, windows of
//                       kept states, short portions, and fp32 models.
//   scan_norm_kernel    the norm and gates behind the scan; puts the tick's last convolution inputs into the ring.
//
// States: [slot][plane][record]; a layer's record holds S [heads, dk, dv], then (mLSTM) n [heads, slices, dk] and m [heads, slices],
// once per slice of 32 value columns.  cur[slot]
// is the live plane; a sequence with its keep flag set stores the state after token j in plane j instead of the live one.
// Gates, decays, state and sums are fp32 throughout.
// Reference parity: the reference's recurrence is Gated DeltaNet only (no counterpart).
#include "scan.cuh"

namespace {

enum { CONV_SILU = 1, CONV_ADD = 2 };                         // silu of the sum; the input itself joins the sum

// thread = one chunk of channels of one token
template <typename T>
__global__ void __launch_bounds__(128)
scan_conv_kernel(const T* proj, int ldp, const float* __restrict__ w, const float* __restrict__ bias, const float* __restrict__ pre,
                 const T* ring, long ring_slot, int ring_rows, int ring_ld, const int* positions, const int* seq_ids,
                 const int* q_start, const int* slots, T* out, int channels, int taps, int mode) {
  constexpr int C = Chunk<T>::N;
  pdl_launch_dependents(40);
  pdl_wait();
  const int t = blockIdx.x, c = (blockIdx.y * 128 + threadIdx.x) * C;
  if (c >= channels) return;
  const int pos = positions[t], seq = seq_ids[t], t0 = q_start[seq];
  const T* rg = ring + (size_t)slots[seq] * ring_slot;
  float acc[C];
#pragma unroll
  for (int e = 0; e < C; ++e) acc[e] = 0.f;
  if (bias) {
#pragma unroll
    for (int e = 0; e < C; e += 4) {
      const float4 b = *reinterpret_cast<const float4*>(bias + c + e);
      acc[e] = b.x, acc[e + 1] = b.y, acc[e + 2] = b.z, acc[e + 3] = b.w;
    }
  }
  for (int j = 0; j < taps; ++j) {            // the last tap multiplies the token's own row
    const int back = taps - 1 - j;
    if (back > pos) continue;
    const T* src = t - back >= t0 ? proj + (size_t)(t - back) * ldp + c : rg + (size_t)((pos - back) % ring_rows) * ring_ld + c;
    float f[C];
    Chunk<T>::get(*reinterpret_cast<const uint4*>(src), f);
    if (pre) {
#pragma unroll
      for (int e = 0; e < C; ++e) f[e] += pre[c + e];
    }
    if ((mode & CONV_ADD) && back == 0) {
#pragma unroll
      for (int e = 0; e < C; ++e) acc[e] += f[e];
    }
#pragma unroll
    for (int e = 0; e < C; e += 4) {
      const float4 b = *reinterpret_cast<const float4*>(w + (size_t)j * channels + c + e);
      acc[e] = fmaf(f[e], b.x, acc[e]), acc[e + 1] = fmaf(f[e + 1], b.y, acc[e + 1]);
      acc[e + 2] = fmaf(f[e + 2], b.z, acc[e + 2]), acc[e + 3] = fmaf(f[e + 3], b.w, acc[e + 3]);
    }
  }
  if (mode & CONV_SILU) {
#pragma unroll
    for (int e = 0; e < C; ++e) acc[e] *= sigmoid_x(acc[e]);
  }
  *reinterpret_cast<uint4*>(out + (size_t)t * channels + c) = Chunk<T>::put(acc);
}

// The same for prompts: thread = one chunk of channels of CR_RUN consecutive tokens; weights and the last inputs stay in registers.
constexpr int CR_RUN = 16;
template <typename T, int K>
__global__ void __launch_bounds__(128)
conv_run_kernel(const T* proj, int ldp, const float* __restrict__ w, const float* __restrict__ bias, const float* __restrict__ pre,
                const T* ring, long ring_slot, int ring_rows, int ring_ld, const int* positions, const int* seq_ids,
                const int* q_start, const int* slots, T* out, int n_tok, int channels, int taps, int mode) {
  constexpr int C = Chunk<T>::N;
  pdl_launch_dependents(44);
  const int c = (blockIdx.y * 128 + threadIdx.x) * C, first = blockIdx.x * CR_RUN, end = min(n_tok, first + CR_RUN);
  if (c >= channels) {
    pdl_wait();
    return;
  }
  float wt[K][C], b[C], p[C], h[K][C];       // weight and input of `k` tokens back (inputs with their bias)
#pragma unroll
  for (int e = 0; e < C; ++e) b[e] = bias ? bias[c + e] : 0.f, p[e] = pre ? pre[c + e] : 0.f;
#pragma unroll
  for (int k = 0; k < K; ++k)
#pragma unroll
    for (int e = 0; e < C; ++e) wt[k][e] = k < taps ? w[(size_t)(taps - 1 - k) * channels + c + e] : 0.f, h[k][e] = 0.f;
  pdl_wait();
  int seq = -1;
#pragma unroll 4
  for (int t = first; t < end; ++t) {
    const uint4 own = *reinterpret_cast<const uint4*>(proj + (size_t)t * ldp + c);
    if (seq_ids[t] != seq) {                 // another sequence (or the run's first token): inputs before this token
      seq = seq_ids[t];
      const int pos = positions[t], t0 = q_start[seq];
      const T* rg = ring + (size_t)slots[seq] * ring_slot + c;
#pragma unroll
      for (int k = 1; k < K; ++k) {
        const bool there = k < taps && k <= pos;
        float f[C];
        if (there) Chunk<T>::get(*reinterpret_cast<const uint4*>(t - k >= t0 ? proj + (size_t)(t - k) * ldp + c : rg + (size_t)((pos - k) % ring_rows) * ring_ld), f);
#pragma unroll
        for (int e = 0; e < C; ++e) h[k][e] = there ? f[e] + p[e] : 0.f;
      }
    }
    Chunk<T>::get(own, h[0]);
    float acc[C];
#pragma unroll
    for (int e = 0; e < C; ++e) {
      h[0][e] += p[e];
      acc[e] = b[e] + (mode & CONV_ADD ? h[0][e] : 0.f);
    }
#pragma unroll
    for (int k = K - 1; k >= 0; --k)
#pragma unroll
      for (int e = 0; e < C; ++e) acc[e] = fmaf(h[k][e], wt[k][e], acc[e]);
#pragma unroll
    for (int k = K - 1; k > 0; --k)
#pragma unroll
      for (int e = 0; e < C; ++e) h[k][e] = h[k - 1][e];
    if (mode & CONV_SILU) {
#pragma unroll
      for (int e = 0; e < C; ++e) acc[e] *= sigmoid_x(acc[e]);
    }
    *reinterpret_cast<uint4*>(out + (size_t)t * channels + c) = Chunk<T>::put(acc);
  }
}

// one block per token: its row into the ring unless later ones of the tick would overwrite it
__global__ void __launch_bounds__(128)
ring_store_kernel(const unsigned char* rows, long ld, unsigned char* ring, long ring_slot, int ring_rows, long ring_ld, int chunks,
                  const int* positions, const int* seq_ids, const int* q_start, const int* q_len, const int* slots) {
  pdl_launch_dependents(43);
  pdl_wait();
  const int t = blockIdx.x, seq = seq_ids[t], left = q_start[seq] + q_len[seq] - 1 - t;
  if (left < 0 || left >= ring_rows) return;
  const uint4* src = reinterpret_cast<const uint4*>(rows + (size_t)t * ld);
  uint4* dst = reinterpret_cast<uint4*>(ring + (size_t)slots[seq] * ring_slot + (size_t)(positions[t] % ring_rows) * ring_ld);
  for (int c = threadIdx.x; c < chunks; c += 128) dst[c] = src[c];
}

// grid (heads * column slices, sequences), 256 threads: lane = column, warp = dk / 8 state rows.  CONV: one token per
// sequence whose rows still have to pass the convolution.  The state is fetched before the dependency wait: its last writer
// is the previous tick, and every tick has launches in between that let their dependents in only after their own wait.
constexpr int SS_TB = 16;
template <typename T, int KIND, int RMAX, bool CONV>
__global__ void __launch_bounds__(256, RMAX <= 16 ? 4 : 2) scan_serial_kernel(const ScanArgs a) {
  constexpr int DK = RMAX * 8;
  __shared__ float s_q[SS_TB][DK], s_k[SS_TB][DK], s_v[SS_TB][32];
  __shared__ float s_keep[SS_TB], s_add[SS_TB], s_floor[SS_TB], s_m;
  __shared__ float s_part[2][8][32], s_den[2][8];
  pdl_launch_dependents(41);
  const int n_sl = (a.dv + 31) / 32, h = blockIdx.x / n_sl, col0 = (blockIdx.x % n_sl) * 32, seq = blockIdx.y;
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
  const int copy = h * n_sl + blockIdx.x % n_sl;            // every slice has its own n and m: they are read and written by it alone
  const size_t n_off = (size_t)a.heads * a.dk * a.dv + (size_t)copy * a.dk + warp * R + lane;
  const size_t m_off = (size_t)a.heads * a.dk * (a.dv + n_sl) + copy;
  float S[RMAX], n = 0.f;
  {
    const float* src = rec + (size_t)plane * a.plane_stride;
#pragma unroll
    for (int r = 0; r < RMAX; ++r) S[r] = r < R && col < a.dv ? src[s_off + (size_t)r * a.dv] : 0.f;
    if (KIND == SCAN_MLSTM) {
      if (lane < R) n = src[n_off];
      if (tid == 0) s_m = src[m_off];
    }
  }
  pdl_wait();
  auto save = [&](int pl) {
    float* dst = rec + (size_t)pl * a.plane_stride;
#pragma unroll
    for (int r = 0; r < RMAX; ++r)
      if (r < R && col < a.dv) dst[s_off + (size_t)r * a.dv] = S[r];
    if (KIND == SCAN_MLSTM && lane < R) dst[n_off] = n;
  };
  const T* base = reinterpret_cast<const T*>(a.rows);
  for (int i0 = 0; i0 < T_; i0 += SS_TB) {
    const int nb = min(SS_TB, T_ - i0);
    __syncthreads();
    if constexpr (CONV) {
      const int pos = a.positions[t0];
      const T* row = base + (size_t)t0 * a.ld;
      const T* rg = reinterpret_cast<const T*>(a.ring) + (size_t)slot * a.ring_slot;
      for (int x = tid; x < 2 * a.dk + 32; x += 256) {
        const int d = x < a.dk ? x : x < 2 * a.dk ? x - a.dk : x - 2 * a.dk;
        const int c = (x < a.dk ? a.q0 : a.k0) + (h / a.per) * a.dk + d, cc = x < 2 * a.dk ? c : a.v0 + h * a.dv + col0 + d;
        float v = 0.f;
        if (x < 2 * a.dk || col0 + d < a.dv) {
          v = a.conv_b[cc];
#pragma unroll 4
          for (int j = 0; j < a.taps; ++j) {
            const int back = a.taps - 1 - j;
            if (back <= pos)
              v = fmaf(to_f(back ? rg[(size_t)((pos - back) % a.ring_rows) * a.ring_ld + cc] : row[cc]), a.conv_w[(size_t)j * a.channels + cc], v);
          }
          v = to_f(from_f<T>(v * sigmoid_x(v)));
        }
        if (x < a.dk) s_q[0][d] = v * a.q_scale;
        else if (x < 2 * a.dk) s_k[0][d] = v;
        else s_v[0][d] = v;
      }
    }
    for (int x = tid; x < (CONV ? 0 : nb * a.dk); x += 256) {
      const int j = x / a.dk, d = x % a.dk;
      const T* row = base + (size_t)(t0 + i0 + j) * a.ld;
      s_q[j][d] = to_f(row[a.q0 + (h / a.per) * a.dk + d]) * a.q_scale;
      s_k[j][d] = to_f(row[a.k0 + (h / a.per) * a.dk + d]);
    }
    for (int x = tid; x < (CONV ? 0 : nb * 32); x += 256)
      s_v[x >> 5][x & 31] = col0 + (x & 31) < a.dv ? to_f(base[(size_t)(t0 + i0 + (x >> 5)) * a.ld + a.v0 + h * a.dv + col0 + (x & 31)]) : 0.f;
    if (tid < nb) {
      float g0, g1;
      scan_gates<KIND>(a, t0 + i0 + tid, h, g0, g1);
      s_keep[tid] = g0, s_add[tid] = g1;
    }
    __syncthreads();
    if (KIND == SCAN_MLSTM) {                  // (f, i) -> factors along the running maximum
      if (tid == 0) {
        float m = s_m;
        for (int j = 0; j < nb; ++j) {
          const float f = s_keep[j], i = s_add[j], now = fmaxf(f + m, i);
          s_keep[j] = expf(f + m - now), s_add[j] = expf(i - now), s_floor[j] = expf(-now);
          m = now;
          if (keep_all) rec[(size_t)(i0 + j) * a.plane_stride + m_off] = m;
        }
        s_m = m;
      }
      __syncthreads();
    }
    for (int j = 0; j < nb; ++j) {
      const float keep = s_keep[j], add = s_add[j], av = add * s_v[j][lane];
      const float *kr = &s_k[j][warp * R], *qr = &s_q[j][warp * R];
      float o = 0.f;
#pragma unroll
      for (int r = 0; r < RMAX; ++r) {
        if (r < R) {
          S[r] = fmaf(kr[r], av, keep * S[r]);
          o = fmaf(qr[r], S[r], o);
        }
      }
      s_part[j & 1][warp][lane] = o;
      if (KIND == SCAN_MLSTM) {
        float d = 0.f;
        if (lane < R) n = fmaf(add, kr[lane], keep * n), d = n * qr[lane];
        d = warp_sum(d);
        if (lane == 0) s_den[j & 1][warp] = d;
      }
      if (keep_all) save(i0 + j);
      __syncthreads();
      if (warp == 0 && col < a.dv) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < 8; ++w) v += s_part[j & 1][w][lane];
        if (KIND == SCAN_MLSTM) {
          float d = 0.f;
#pragma unroll
          for (int w = 0; w < 8; ++w) d += s_den[j & 1][w];
          v /= fmaxf(fabsf(d), s_floor[j]) + 1e-6f;
        } else if (KIND == SCAN_MAMBA2) {
          v = fmaf(a.skip[h], s_v[j][lane], v);
        }
        a.o[((size_t)(t0 + i0 + j) * a.heads + h) * a.dv + col] = v;
      }
    }
  }
  if (!keep_all) {
    save(plane);
    if (KIND == SCAN_MLSTM && tid == 0) rec[(size_t)plane * a.plane_stride + m_off] = s_m;
  }
}

struct NormArgs {
  const float* o;              // [T, heads * dv]
  const void* gate;            // gate columns of the fused projection rows
  int ldp;
  const float* w;
  void* out;
  int n_out, heads, vdim, dv, groups;
  float eps;
  // convolution inputs of the tick's last tokens into the ring (Mamba-2)
  const void* conv_in;
  void* ring;
  long ring_slot;
  int ring_rows, ring_ld, channels;
  const int *positions, *seq_ids, *q_start, *q_len, *slots;
};

// gates behind a recurrence's norm
template <typename T> __device__ __forceinline__ float gate_x(float z) { return sizeof(T) == 2 ? sigmoid_f(z) : sigmoid_x(z); }

// one block per token; NORM_R: float4 a thread keeps of a row
template <typename T, int KIND, int NORM_R>
__global__ void __launch_bounds__(256) scan_norm_kernel(const NormArgs a) {
  extern __shared__ float s_y[];               // [heads * vdim], true columns only
  __shared__ float red[32];
  constexpr int C = Chunk<T>::N;
  pdl_launch_dependents(42);
  pdl_wait();
  const int t = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, inner = a.heads * a.vdim;
  const float* o = a.o + (size_t)t * a.heads * a.dv;
  const T* gate = reinterpret_cast<const T*>(a.gate) + (size_t)t * a.ldp;
  if (KIND == SCAN_MAMBA2) {
    const int seq = a.seq_ids[t], left = a.q_start[seq] + a.q_len[seq] - 1 - t;
    if (left >= 0 && left < a.ring_rows) {
      const uint4* src = reinterpret_cast<const uint4*>(reinterpret_cast<const T*>(a.conv_in) + (size_t)t * a.ldp);
      uint4* dst = reinterpret_cast<uint4*>(reinterpret_cast<T*>(a.ring) + (size_t)a.slots[seq] * a.ring_slot +
                                            (size_t)(a.positions[t] % a.ring_rows) * a.ring_ld);
      for (int c = tid; c < a.channels / C; c += 256) dst[c] = src[c];
    }
  }
  T* out = reinterpret_cast<T*>(a.out) + (size_t)t * a.n_out;
  if (a.vdim == a.dv && inner % 1024 == 0 && inner <= NORM_R * 1024 && (inner / a.groups) % 128 == 0) {
    // unpadded heads, groups of whole warps of four columns a thread: everything stays in registers
    float4 v[NORM_R], z[NORM_R];
    const int nr = inner / 1024;
#pragma unroll
    for (int i = 0; i < NORM_R; ++i)
      if (i < nr) v[i] = *reinterpret_cast<const float4*>(o + (i * 256 + tid) * 4), z[i] = load4(gate + (i * 256 + tid) * 4);
#pragma unroll
    for (int i = 0; i < NORM_R; ++i)
      if (i < nr) {
        const float4 s = make_float4(gate_x<T>(z[i].x), gate_x<T>(z[i].y), gate_x<T>(z[i].z), gate_x<T>(z[i].w));
        if (KIND == SCAN_MAMBA2) v[i].x *= z[i].x * s.x, v[i].y *= z[i].y * s.y, v[i].z *= z[i].z * s.z, v[i].w *= z[i].w * s.w;
        z[i] = s;
        const float ss = warp_sum(v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w);
        if (lane == 0) s_y[i * 8 + warp] = ss;             // sums of 128 columns each
      }
    __syncthreads();
    const int per = inner / a.groups / 128;
#pragma unroll
    for (int i = 0; i < NORM_R; ++i)
      if (i < nr) {
        const int g = (i * 8 + warp) / per, p = (i * 256 + tid) * 4;
        float ss = 0.f;
        for (int k = 0; k < per; ++k) ss += s_y[g * per + k];
        const float r = inv_rms(ss, per * 128, a.eps);
        const float4 w = *reinterpret_cast<const float4*>(a.w + p);
        float4 y = make_float4(v[i].x * r * w.x, v[i].y * r * w.y, v[i].z * r * w.z, v[i].w * r * w.w);
        if (KIND == SCAN_MLSTM) y.x *= z[i].x, y.y *= z[i].y, y.z *= z[i].z, y.w *= z[i].w;
        store4<T>(out + p, y.x, y.y, y.z, y.w);
      }
    for (int p = inner + tid; p < a.n_out; p += 256) out[p] = from_f<T>(0.f);
    return;
  }
  for (int x = tid; x < inner; x += 256) {
    const int p = x / a.vdim * a.dv + x % a.vdim;
    float v = o[p];
    if (KIND == SCAN_MAMBA2) {
      const float z = to_f(gate[p]);
      v *= z * sigmoid_x(z);
    }
    s_y[x] = v;
  }
  __syncthreads();
  const int gs = inner / a.groups;
  if (a.groups >= 8) {
    for (int g = warp; g < a.groups; g += 8) {
      float ss = 0.f;
      for (int x = lane; x < gs; x += 32) ss += s_y[g * gs + x] * s_y[g * gs + x];
      const float r = inv_rms(warp_sum(ss), gs, a.eps);
      for (int x = lane; x < gs; x += 32) s_y[g * gs + x] *= r;
    }
  } else {
    for (int g = 0; g < a.groups; ++g) {
      float ss = 0.f;
      for (int x = tid; x < gs; x += 256) ss += s_y[g * gs + x] * s_y[g * gs + x];
      const float r = inv_rms(block_sum(ss, red), gs, a.eps);
      for (int x = tid; x < gs; x += 256) s_y[g * gs + x] *= r;
    }
  }
  __syncthreads();
  for (int p = tid; p < a.n_out; p += 256) {
    const int h = p / a.dv, d = p % a.dv;
    float v = 0.f;
    if (h < a.heads && d < a.vdim) {
      v = s_y[h * a.vdim + d] * a.w[p];
      if (KIND == SCAN_MLSTM) v *= sigmoid_x(to_f(gate[p]));
    }
    out[p] = from_f<T>(v);
  }
}

template <typename T, int KIND, bool CONV>
cudaError_t serial_launch(const ScanArgs& a, int B, cudaStream_t st) {
  const dim3 grid(a.heads * ((a.dv + 31) / 32), B);
  if (a.dk <= 32) return trl_launch(scan_serial_kernel<T, KIND, 4, CONV>, grid, dim3(256), 0, st, a);
  if (a.dk <= 64) return trl_launch(scan_serial_kernel<T, KIND, 8, CONV>, grid, dim3(256), 0, st, a);
  if (a.dk <= 128) return trl_launch(scan_serial_kernel<T, KIND, 16, CONV>, grid, dim3(256), 0, st, a);
  return trl_launch(scan_serial_kernel<T, KIND, 32, CONV>, grid, dim3(256), 0, st, a);
}

}  // namespace

// The last rows of every sequence's tick into its ring: `channels` columns from rows (leading dimension ld, bytes per value: item).
TRL_API int trl_ring_store(const void* rows, int ld, void* ring, long ring_slot, int ring_rows, int ring_ld, int channels, const void* positions,
                           const void* seq_ids, const void* q_start, const void* q_len, const void* slots, int T, int f32, void* stream) {
  const int item = f32 ? 4 : 2, per = 16 / item;
  if (T <= 0 || channels <= 0 || channels % per || ld % per || ring_ld % per || ring_slot % per || ring_rows <= 0 || ((uintptr_t)ring & 15) ||
      ((uintptr_t)rows & 15))
    return (int)cudaErrorInvalidValue;
  return (int)trl_launch(ring_store_kernel, dim3(T), dim3(128), 0, (cudaStream_t)stream, (const unsigned char*)rows, (long)ld * item,
                         (unsigned char*)ring, ring_slot * item, ring_rows, (long)ring_ld * item, channels / per, (const int*)positions,
                         (const int*)seq_ids, (const int*)q_start, (const int*)q_len, (const int*)slots);
}

// proj: rows whose first `channels` columns are convolved; w: [taps, channels]; pre (or null): bias of the inputs, which zeros before
// a sequence's start do not get; bias may be null; mode: CONV_* bits; ring: the layer's first column of slot 0.
TRL_API int trl_scan_conv(const void* proj, int ldp, const void* w, const void* bias, const void* pre, const void* ring, long ring_slot,
                          int ring_rows, int ring_ld, const void* positions, const void* seq_ids, const void* q_start, const void* slots,
                          void* out, int T, int channels, int taps, int mode, int f32, void* stream) {
  const int per = f32 ? 4 : 8;
  if (T <= 0 || channels <= 0 || channels % 16 || taps < 1 || taps > ring_rows || ldp % per || ring_ld % per || ring_slot % per ||
      ((uintptr_t)ring & 15) || ((uintptr_t)proj & 15))
    return (int)cudaErrorInvalidValue;
  const dim3 grid(T, (channels / per + 127) / 128);
  if (T >= 512 && taps <= 4) {
    const dim3 runs((T + CR_RUN - 1) / CR_RUN, grid.y);
#define CONV_RUN(TT)                                                                                                               \
  return (int)trl_launch(conv_run_kernel<TT, 4>, runs, dim3(128), 0, (cudaStream_t)stream, (const TT*)proj, ldp, (const float*)w,  \
                         (const float*)bias, (const float*)pre, (const TT*)ring, ring_slot, ring_rows, ring_ld, (const int*)positions, \
                         (const int*)seq_ids, (const int*)q_start, (const int*)slots, (TT*)out, T, channels, taps, mode)
    if (f32) CONV_RUN(float);
    CONV_RUN(bf16);
#undef CONV_RUN
  }
  if (f32)
    return (int)trl_launch(scan_conv_kernel<float>, grid, dim3(128), 0, (cudaStream_t)stream, (const float*)proj, ldp, (const float*)w,
                           (const float*)bias, (const float*)pre, (const float*)ring, ring_slot, ring_rows, ring_ld, (const int*)positions,
                           (const int*)seq_ids, (const int*)q_start, (const int*)slots, (float*)out, channels, taps, mode);
  return (int)trl_launch(scan_conv_kernel<bf16>, grid, dim3(128), 0, (cudaStream_t)stream, (const bf16*)proj, ldp, (const float*)w,
                         (const float*)bias, (const float*)pre, (const bf16*)ring, ring_slot, ring_rows, ring_ld, (const int*)positions,
                         (const int*)seq_ids, (const int*)q_start, (const int*)slots, (bf16*)out, channels, taps, mode);
}

// kind: SCAN_*.  args: a ScanArgs (scan.cuh) filled by the caller.  Serves sequences of min_len..max_len tokens.
TRL_API int trl_scan_serial(const ScanArgs* a, int B, int kind, int f32, void* stream) {
  if (B <= 0 || scan_args_bad(*a, kind) || (a->taps && (kind != SCAN_MAMBA2 || a->taps > a->ring_rows || !a->conv_w || !a->conv_b || !a->ring ||
                                                        !a->positions || a->keep_flags)))
    return (int)cudaErrorInvalidValue;
  cudaStream_t st = (cudaStream_t)stream;
  if (kind == SCAN_MAMBA2 && a->taps)
    return (int)(f32 ? serial_launch<float, SCAN_MAMBA2, true>(*a, B, st) : serial_launch<bf16, SCAN_MAMBA2, true>(*a, B, st));
  if (kind == SCAN_MAMBA2)
    return (int)(f32 ? serial_launch<float, SCAN_MAMBA2, false>(*a, B, st) : serial_launch<bf16, SCAN_MAMBA2, false>(*a, B, st));
  if (kind == SCAN_FIXED) return (int)(f32 ? serial_launch<float, SCAN_FIXED, false>(*a, B, st) : serial_launch<bf16, SCAN_FIXED, false>(*a, B, st));
  return (int)(f32 ? serial_launch<float, SCAN_MLSTM, false>(*a, B, st) : serial_launch<bf16, SCAN_MLSTM, false>(*a, B, st));
}

// o: fp32 [T, heads * dv]; gate, conv_in: columns of the fused projection rows (ldp wide); out: [T, n_out].
TRL_API int trl_scan_norm(const void* o, const void* gate, int ldp, const void* w, void* out, int n_out, int T, int heads, int vdim, int dv,
                          int groups, float eps, const void* conv_in, void* ring, long ring_slot, int ring_rows, int ring_ld, int channels,
                          const void* positions, const void* seq_ids, const void* q_start, const void* q_len, const void* slots, int kind,
                          int f32, void* stream) {
  const int per = f32 ? 4 : 8;
  const size_t smem = (size_t)heads * vdim * sizeof(float);
  if (T <= 0 || heads <= 0 || vdim > dv || groups <= 0 || (heads * vdim) % groups || n_out < heads * dv || smem > 160 * 1024 ||
      (kind == SCAN_MAMBA2 && (!ring || channels % 16 || ring_ld % per || ring_slot % per || ldp % per)))
    return (int)cudaErrorInvalidValue;
  NormArgs a;
  a.o = (const float*)o, a.gate = gate, a.ldp = ldp, a.w = (const float*)w, a.out = out, a.n_out = n_out, a.heads = heads, a.vdim = vdim;
  a.dv = dv, a.groups = groups, a.eps = eps, a.conv_in = conv_in, a.ring = ring, a.ring_slot = ring_slot, a.ring_rows = ring_rows;
  a.ring_ld = ring_ld, a.channels = channels, a.positions = (const int*)positions, a.seq_ids = (const int*)seq_ids;
  a.q_start = (const int*)q_start, a.q_len = (const int*)q_len, a.slots = (const int*)slots;
  cudaStream_t st = (cudaStream_t)stream;
#define NORM_AS(TT, KK)                                                                                                    \
  if (heads * vdim <= 4096) NORM_R_AS(TT, KK, 4)                                                                           \
  else NORM_R_AS(TT, KK, 8)
#define NORM_R_AS(TT, KK, RR)                                                                                              \
  {                                                                                                                        \
    auto k = scan_norm_kernel<TT, KK, RR>;                                                                                     \
    static bool configured = false;                                                                                        \
    if (!configured) {                                                                                                     \
      const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);              \
      if (e != cudaSuccess) return (int)e;                                                                                 \
      configured = true;                                                                                                   \
    }                                                                                                                      \
    return (int)trl_launch(k, dim3(T), dim3(256), smem, st, a);                                                            \
  }
  if (kind == SCAN_MAMBA2) {
    if (f32) NORM_AS(float, SCAN_MAMBA2)
    NORM_AS(bf16, SCAN_MAMBA2)
  }
  if (f32) NORM_AS(float, SCAN_MLSTM)
  NORM_AS(bf16, SCAN_MLSTM)
#undef NORM_AS
#undef NORM_R_AS
}
