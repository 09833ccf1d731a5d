// Latent attention around its attention kernels: what a token writes to the cache, its rotated queries, the gated output,
// and the attention itself in its plain form.
//
// The cache holds one row per token, [latent | rotated shared key], in packed pages (tilerl_b200/kv.py, LatentPage).
// Queries are mapped into the latent (W_uk^T q per head), so every head reads the same rows, and the weighted sum of
// latents is mapped back (W_uv per head) afterwards.
//
//   latent_prep_kernel   per token: RMS-normed query latent; RMS-normed kv latent and rotated key into the page.
//   latent_rope_kernel   the rotated part of every query head, in place.
//   latent_gate_kernel   head outputs times sigmoid(gate), padded to the output projection's columns.
//   latent_attn_kernel   windowed softmax attention on CUDA cores, any size: fp32 models, and shapes without a
//                        tensor-core form (latent_mma.cu).
//
// Angles are formed and reduced in fp64 from the position and the pair's frequency: fp32 products of positions in the
// thousands would already carry 1e-4 radians.
// Reference parity: the reference's attention keeps full keys and values (no counterpart).
#include "packed.cuh"

namespace {

struct PrepArgs {
  int ldp, c0, kr0, q_rank, kv_rank, kv, rd, n_pairs, n_blocks;
  float amp, eps;
};

template <typename T>
__global__ void __launch_bounds__(256)
latent_prep_kernel(const T* proj, const float* __restrict__ q_norm, const float* __restrict__ kv_norm, const double* __restrict__ freqs,
                   const int* positions, const int* slot_mapping, T* cq, unsigned char* pages, const PrepArgs a) {
  constexpr int C = Chunk<T>::N;
  __shared__ float red[32];
  pdl_launch_dependents(33);
  pdl_wait();
  const int t = blockIdx.x;
  const T* row = proj + (size_t)t * a.ldp;
  float f[C];
  const uint4* qs = reinterpret_cast<const uint4*>(row);
  const uint4* ks = reinterpret_cast<const uint4*>(row + a.c0);
  float s1 = 0.f, s2 = 0.f;
  for (int c = threadIdx.x; c < a.c0 / C; c += blockDim.x) {
    Chunk<T>::get(qs[c], f);
#pragma unroll
    for (int i = 0; i < C; ++i) s1 += f[i] * f[i];
  }
  for (int c = threadIdx.x; c < a.kv / C; c += blockDim.x) {
    Chunk<T>::get(ks[c], f);
#pragma unroll
    for (int i = 0; i < C; ++i) s2 += f[i] * f[i];
  }
  const float r1 = inv_rms(block_sum(s1, red), a.q_rank, a.eps), r2 = inv_rms(block_sum(s2, red), a.kv_rank, a.eps);
  uint4* qd = reinterpret_cast<uint4*>(cq + (size_t)t * a.c0);
  for (int c = threadIdx.x; c < a.c0 / C; c += blockDim.x) {
    Chunk<T>::get(qs[c], f);
#pragma unroll
    for (int i = 0; i < C; ++i) f[i] = f[i] * r1 * q_norm[c * C + i];
    qd[c] = Chunk<T>::put(f);
  }
  int slot = slot_mapping[t];
  if (slot < 0) return;
  slot = trl_checked(slot, a.n_blocks * KVB, 9);
  const int r = slot % KVB, n_ch = (a.kv + a.rd) / C, n_kv = a.kv / C;
  uint4* dst = reinterpret_cast<uint4*>(pages + (size_t)(slot / KVB) * n_ch * 16 * KVB) + r * n_ch;
  const int pos = positions[t];
  for (int c = threadIdx.x; c < n_ch; c += blockDim.x) {
    if (c < n_kv) {
      Chunk<T>::get(ks[c], f);
#pragma unroll
      for (int i = 0; i < C; ++i) f[i] = f[i] * r2 * kv_norm[c * C + i];
    } else {
      Chunk<T>::get(reinterpret_cast<const uint4*>(row + a.kr0)[c - n_kv], f);
#pragma unroll
      for (int i = 0; i < C; i += 2) {
        const int p = ((c - n_kv) * C + i) / 2;
        if (p < a.n_pairs) {
          float cs, sn;
          pair_angle(pos, freqs[p], a.amp, cs, sn);
          const float u = f[i], v = f[i + 1];
          f[i] = u * cs - v * sn, f[i + 1] = v * cs + u * sn;
        }
      }
    }
    dst[page_chunk(c, r, n_ch)] = Chunk<T>::put(f);
  }
}

template <typename T>
__global__ void __launch_bounds__(128)
latent_rope_kernel(T* q, const double* __restrict__ freqs, const int* positions, int heads, int dq, int dk, int n_pairs, float amp) {
  extern __shared__ float2 cs[];
  pdl_launch_dependents(34);
  pdl_wait();
  const int t = blockIdx.x, pos = positions[t];
  for (int p = threadIdx.x; p < n_pairs; p += blockDim.x) pair_angle(pos, freqs[p], amp, cs[p].x, cs[p].y);
  __syncthreads();
  for (int x = threadIdx.x; x < heads * n_pairs; x += blockDim.x) {
    const int h = x / n_pairs, p = x % n_pairs;
    T* d = q + ((size_t)t * heads + h) * dq + dk + 2 * p;
    const float u = to_f(d[0]), v = to_f(d[1]);
    d[0] = from_f<T>(u * cs[p].x - v * cs[p].y), d[1] = from_f<T>(v * cs[p].x + u * cs[p].y);
  }
}

// o: [heads, T, dv] (head-major); gate: the gate columns of the fused projection rows
template <typename T>
__global__ void __launch_bounds__(256)
latent_gate_kernel(const T* o, const T* gate, int ldp, T* out, int n_out, int n_tok, int heads, int dv) {
  constexpr int C = Chunk<T>::N;
  pdl_launch_dependents(35);
  pdl_wait();
  const int t = blockIdx.x;
  for (int c = threadIdx.x; c < n_out / C; c += blockDim.x) {
    float f[C], g[C];
#pragma unroll
    for (int i = 0; i < C; ++i) f[i] = 0.f;
    const int h = c * C / dv;
    if (h < heads) {
      Chunk<T>::get(*reinterpret_cast<const uint4*>(o + ((size_t)h * n_tok + t) * dv + c * C - h * dv), f);
      Chunk<T>::get(*reinterpret_cast<const uint4*>(gate + (size_t)t * ldp + c * C), g);
#pragma unroll
      for (int i = 0; i < C; ++i) f[i] *= sigmoid_x(g[i]);
    }
    *reinterpret_cast<uint4*>(out + (size_t)t * n_out + c * C) = Chunk<T>::put(f);
  }
}

// One block = (16 rows, sequence); a row is a (token, head) pair.  Thread (r, c) forms the score of row r and key c of a
// page and owns the output columns c, c + 16, ... of row r.
constexpr int F_ROWS = 16, F_MAXKV = 1024;
template <typename T>
__global__ void __launch_bounds__(256)
latent_attn_kernel(const T* ql, long ql_h, long ql_t, const T* q, int dq, int dk, const unsigned char* pages, int kv, int rd, int n_blocks,
                   const int* table, int max_blocks, const int* q_start, const int* q_len, const int* positions, T* oc, long oc_h,
                   long oc_t, int heads, int window, float scale) {
  constexpr int C = Chunk<T>::N;
  extern __shared__ float sf[];
  __shared__ float s_w[F_ROWS][KVB + 1];
  pdl_launch_dependents(36);
  pdl_wait();
  const int seq = blockIdx.y, n_rows = q_len[seq] * heads, row0 = blockIdx.x * F_ROWS;
  if (row0 >= n_rows) return;
  const int q0 = q_start[seq], D = kv + rd, n_ch = D / C;
  float* sq = sf;                                  // [16][D + 1]
  float* sk = sq + F_ROWS * (D + 1);               // [16][D + 1]
  const int r = threadIdx.x >> 4, c = threadIdx.x & 15, row = row0 + r;
  const bool in = row < n_rows;
  const int t = q0 + (in ? row / heads : 0), h = in ? row % heads : 0;
  for (int d = c; d < D; d += 16) {
    float v = 0.f;
    if (in) v = d < kv ? to_f(ql[h * ql_h + t * ql_t + d]) : to_f(q[((size_t)t * heads + h) * dq + dk + d - kv]);
    sq[r * (D + 1) + d] = v;
  }
  const int pos = in ? positions[t] : -1;
  const int last = positions[q0 + (min(row0 + F_ROWS, n_rows) - 1) / heads], first = max(0, positions[q0 + row0 / heads] - window + 1);
  float acc[F_MAXKV / 16], top = -INFINITY, sum = 0.f;
#pragma unroll
  for (int i = 0; i < F_MAXKV / 16; ++i) acc[i] = 0.f;
  for (int p = first / KVB; p * KVB <= last; ++p) {
    const int blk = trl_checked(table[(size_t)seq * max_blocks + p], n_blocks, 10);
    const uint4* page = reinterpret_cast<const uint4*>(pages + (size_t)blk * n_ch * 16 * KVB);
    __syncthreads();
    for (int x = threadIdx.x; x < KVB * n_ch; x += 256) {
      const int kr = x / n_ch, cc = x % n_ch;
      float f[C];
#pragma unroll
      for (int i = 0; i < C; ++i) f[i] = 0.f;
      if (p * KVB + kr <= last) Chunk<T>::get(page[kr * n_ch + page_chunk(cc, kr, n_ch)], f);
#pragma unroll
      for (int i = 0; i < C; ++i) sk[kr * (D + 1) + cc * C + i] = f[i];
    }
    __syncthreads();
    float s = 0.f;
    for (int d = 0; d < D; ++d) s = fmaf(sq[r * (D + 1) + d], sk[c * (D + 1) + d], s);
    const int j = p * KVB + c;
    s = j <= pos && pos - j < window ? s * scale : -INFINITY;
    float m = s;
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
    const float now = fmaxf(top, m);
    // (no branch: the two rows of a warp may differ in whether anything of their window has come by)
    const float ref = now == -INFINITY ? 0.f : now, w = expf(s - ref), back = expf(top - ref);
    s_w[r][c] = w;
    float ws = w;
#pragma unroll
    for (int o = 8; o > 0; o >>= 1) ws += __shfl_xor_sync(0xffffffffu, ws, o);
    sum = sum * back + ws, top = now;
#pragma unroll
    for (int i = 0; i < F_MAXKV / 16; ++i) acc[i] *= back;
    __syncwarp();                                  // a row's 16 threads share a warp
#pragma unroll
    for (int i = 0; i < F_MAXKV / 16; ++i) {
      const int d = c + 16 * i;
      if (d < kv) {
#pragma unroll
        for (int k = 0; k < KVB; ++k) acc[i] = fmaf(s_w[r][k], sk[k * (D + 1) + d], acc[i]);
      }
    }
  }
  if (in)
#pragma unroll
    for (int i = 0; i < F_MAXKV / 16; ++i)
      if (c + 16 * i < kv) oc[h * oc_h + t * oc_t + c + 16 * i] = from_f<T>(acc[i] / sum);
}

}  // namespace

// proj rows [query latent | kv latent | key part | ...]: c0, kr0 = first column of the second and third part.  cq: [T, c0].
// pages: [n_blocks, 16 * (kv + rd)] elements.  freqs: n_pairs doubles.
TRL_API int trl_latent_prep(const void* proj, int ldp, const void* q_norm, const void* kv_norm, const void* freqs, const void* positions,
                            const void* slot_mapping, void* cq, void* pages, int n_blocks, int T, int c0, int kr0, int q_rank,
                            int kv_rank, int kv, int rd, int n_pairs, float amp, float eps, int f32, void* stream) {
  const int per = f32 ? 4 : 8;
  if (T <= 0 || ldp % per || c0 % per || kr0 % per || kv % 16 || rd % 16 || n_pairs * 2 > rd || q_rank > c0 || kv_rank > kv ||
      kr0 + rd > ldp || n_blocks <= 0 || ((uintptr_t)pages & 15))
    return (int)cudaErrorInvalidValue;
  PrepArgs a;
  a.ldp = ldp, a.c0 = c0, a.kr0 = kr0, a.q_rank = q_rank, a.kv_rank = kv_rank, a.kv = kv, a.rd = rd, a.n_pairs = n_pairs;
  a.n_blocks = n_blocks, a.amp = amp, a.eps = eps;
  cudaStream_t st = (cudaStream_t)stream;
  if (f32)
    return (int)trl_launch(latent_prep_kernel<float>, dim3(T), dim3(256), 0, st, (const float*)proj, (const float*)q_norm,
                           (const float*)kv_norm, (const double*)freqs, (const int*)positions, (const int*)slot_mapping, (float*)cq,
                           (unsigned char*)pages, a);
  return (int)trl_launch(latent_prep_kernel<bf16>, dim3(T), dim3(256), 0, st, (const bf16*)proj, (const float*)q_norm,
                         (const float*)kv_norm, (const double*)freqs, (const int*)positions, (const int*)slot_mapping, (bf16*)cq,
                         (unsigned char*)pages, a);
}

// q: [T, heads, dq], the rotated part starts at column dk.
TRL_API int trl_latent_rope(void* q, const void* freqs, const void* positions, int T, int heads, int dq, int dk, int n_pairs, float amp,
                            int f32, void* stream) {
  if (T <= 0 || heads <= 0 || n_pairs <= 0 || dk + 2 * n_pairs > dq || n_pairs > 4096) return (int)cudaErrorInvalidValue;
  const size_t sm = n_pairs * sizeof(float2);
  if (f32)
    return (int)trl_launch(latent_rope_kernel<float>, dim3(T), dim3(128), sm, (cudaStream_t)stream, (float*)q, (const double*)freqs,
                           (const int*)positions, heads, dq, dk, n_pairs, amp);
  return (int)trl_launch(latent_rope_kernel<bf16>, dim3(T), dim3(128), sm, (cudaStream_t)stream, (bf16*)q, (const double*)freqs,
                         (const int*)positions, heads, dq, dk, n_pairs, amp);
}

TRL_API int trl_latent_gate(const void* o, const void* gate, int ldp, void* out, int n_out, int T, int heads, int dv, int f32, void* stream) {
  if (T <= 0 || heads <= 0 || dv % 16 || n_out % 16 || n_out < heads * dv || ldp % (f32 ? 4 : 8)) return (int)cudaErrorInvalidValue;
  if (f32)
    return (int)trl_launch(latent_gate_kernel<float>, dim3(T), dim3(256), 0, (cudaStream_t)stream, (const float*)o, (const float*)gate,
                           ldp, (float*)out, n_out, T, heads, dv);
  return (int)trl_launch(latent_gate_kernel<bf16>, dim3(T), dim3(256), 0, (cudaStream_t)stream, (const bf16*)o, (const bf16*)gate, ldp,
                         (bf16*)out, n_out, T, heads, dv);
}

// ql: latent queries, element (t, h, d) at h * ql_h + t * ql_t + d; oc: latent sums likewise.  q: [T, heads, dq].
TRL_API int trl_latent_attn(const void* ql, long ql_h, long ql_t, const void* q, int dq, int dk, const void* pages, int kv, int rd,
                            int n_blocks, const void* table, int max_blocks, const void* q_start, const void* q_len,
                            const void* positions, void* oc, long oc_h, long oc_t, int B, int max_q_len, int heads, int window,
                            float scale, int f32, void* stream) {
  const size_t smem = (size_t)2 * F_ROWS * (kv + rd + 1) * sizeof(float);
  if (B <= 0 || max_q_len <= 0 || heads <= 0 || kv % 16 || rd % 16 || kv <= 0 || kv > F_MAXKV || dk + rd > dq || window <= 0 ||
      n_blocks <= 0 || smem > 200 * 1024)
    return (int)cudaErrorInvalidValue;
  static bool configured = false;
  if (!configured) {
    cudaError_t e = cudaFuncSetAttribute(latent_attn_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(latent_attn_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
    if (e != cudaSuccess) return (int)e;
    configured = true;
  }
  const dim3 grid((max_q_len * heads + F_ROWS - 1) / F_ROWS, B);
  if (f32)
    return (int)trl_launch(latent_attn_kernel<float>, grid, dim3(256), smem, (cudaStream_t)stream, (const float*)ql, ql_h, ql_t,
                           (const float*)q, dq, dk, (const unsigned char*)pages, kv, rd, n_blocks, (const int*)table, max_blocks,
                           (const int*)q_start, (const int*)q_len, (const int*)positions, (float*)oc, oc_h, oc_t, heads, window, scale);
  return (int)trl_launch(latent_attn_kernel<bf16>, grid, dim3(256), smem, (cudaStream_t)stream, (const bf16*)ql, ql_h, ql_t,
                         (const bf16*)q, dq, dk, (const unsigned char*)pages, kv, rd, n_blocks, (const int*)table, max_blocks,
                         (const int*)q_start, (const int*)q_len, (const int*)positions, (bf16*)oc, oc_h, oc_t, heads, window, scale);
}
