// fp32 residual stream of parallel-block decoders (models/zinutar.py): embedding + norm, norm of the stream
// into a projection's input, stream addition, and the middle of a block, which takes the fused projection
// rows [q | k | v | up] apart: K / V into the packed pages (layout: tilerl_b200/kv.py, KvPage) and
// PolyNorm(up) into the feed-forward columns of the output projection's input.
// Stream rows are `ld` wide (a multiple of 64) with zeros past the model width `n`.
// Reference parity: the reference keeps a bf16 residual and has no PolyNorm (no counterpart).
#include "packed.cuh"

namespace {

constexpr int RMS_BYTES = 128;

// x = rms(table[id]) * w, optionally kept a second time (the embedding output re-entering a loop)
template <typename T>
__global__ void __launch_bounds__(256)
embed_norm_kernel(const T* __restrict__ table, const int* ids, const float* __restrict__ w, float* x, float* keep, int ld,
                  int n, int V, float eps) {
  constexpr int C = Chunk<T>::N;
  __shared__ float red[32];
  pdl_launch_dependents(20);
  pdl_wait();
  const int t = blockIdx.x, id = ids[t];
  float* xr = x + (size_t)t * ld;
  float* kr = keep ? keep + (size_t)t * ld : nullptr;
  if (id < 0 || id >= V) {   // never read outside the table: zero row + error word {BOUNDS, 1, token, id}
    if (threadIdx.x == 0) trl_set_error(TRL_ERR_BOUNDS, 1, t, id);
    for (int i = threadIdx.x; i < ld; i += blockDim.x) {
      xr[i] = 0.f;
      if (kr) kr[i] = 0.f;
    }
    return;
  }
  const uint4* src = reinterpret_cast<const uint4*>(table + (size_t)id * ld);
  float ss = 0.f, f[C];
  for (int c = threadIdx.x; c < ld / C; c += blockDim.x) {
    Chunk<T>::get(src[c], f);
#pragma unroll
    for (int i = 0; i < C; ++i) ss += f[i] * f[i];
  }
  const float r = inv_rms(block_sum(ss, red), n, eps);
  for (int c = threadIdx.x; c < ld / C; c += blockDim.x) {
    Chunk<T>::get(src[c], f);
#pragma unroll
    for (int i = 0; i < C; i += 4) {
      const int k = c * C + i;
      const float4 ww = *reinterpret_cast<const float4*>(w + k);
      const float4 v = make_float4(f[i] * r * ww.x, f[i + 1] * r * ww.y, f[i + 2] * r * ww.z, f[i + 3] * r * ww.w);
      *reinterpret_cast<float4*>(xr + k) = v;
      if (kr) *reinterpret_cast<float4*>(kr + k) = v;
    }
  }
}

// h = rms(x) * w in the projection's input type
template <typename T>
__global__ void __launch_bounds__(256)
stream_norm_kernel(const float* x, const float* __restrict__ w, T* h, int ld, int n, float eps) {
  constexpr int R = 8;                       // float4 a thread keeps in registers (rows up to 8192 wide)
  __shared__ float red[32];
  pdl_launch_dependents(21);
  pdl_wait();
  const float4* xr = reinterpret_cast<const float4*>(x + (size_t)blockIdx.x * ld);
  const float4* wr = reinterpret_cast<const float4*>(w);
  const int nv = ld / 4;
  float4 v[R];
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int c = threadIdx.x + i * 256;
    v[i] = c < nv ? xr[c] : make_float4(0.f, 0.f, 0.f, 0.f);
    ss += v[i].x * v[i].x + v[i].y * v[i].y + v[i].z * v[i].z + v[i].w * v[i].w;
  }
  for (int c = threadIdx.x + R * 256; c < nv; c += 256) {
    const float4 a = xr[c];
    ss += a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w;
  }
  const float r = inv_rms(block_sum(ss, red), n, eps);
  T* hr = h + (size_t)blockIdx.x * ld;
  auto store = [&](int c, const float4& a) {
    const float4 b = wr[c];
    const float y0 = a.x * r * b.x, y1 = a.y * r * b.y, y2 = a.z * r * b.z, y3 = a.w * r * b.w;
    if constexpr (sizeof(T) == 2)
      *reinterpret_cast<uint2*>(hr + c * 4) = make_uint2(f2_to_bf162_bits(y0, y1), f2_to_bf162_bits(y2, y3));
    else
      *reinterpret_cast<float4*>(hr + c * 4) = make_float4(y0, y1, y2, y3);
  };
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int c = threadIdx.x + i * 256;
    if (c < nv) store(c, v[i]);
  }
  for (int c = threadIdx.x + R * 256; c < nv; c += 256) store(c, xr[c]);
}

__global__ void __launch_bounds__(256) stream_add_kernel(float4* x, const float4* y, long n4) {
  pdl_launch_dependents(22);
  pdl_wait();
  for (long i = blockIdx.x * 256L + threadIdx.x; i < n4; i += (long)gridDim.x * 256) {
    float4 a = x[i];
    const float4 b = y[i];
    a.x += b.x, a.y += b.y, a.z += b.z, a.w += b.w;
    x[i] = a;
  }
}

struct MidArgs {
  int ldp, ldm, k0, v0, up0, attn_cols, ff;        // elements
  int n_kv, dim, kch, vch, page_bytes, n_blocks;   // packed page: chunks per K / V row
  float eps;
};

// grid (token, part): part 0 = feed-forward columns, parts 1.. = K / V heads, one warp per head
template <typename T>
__global__ void __launch_bounds__(1024)
block_mid_kernel(const T* proj, const float* __restrict__ act, T* mid, const int* slot_mapping, unsigned char* pages,
                 const MidArgs a) {
  constexpr int C = Chunk<T>::N, R = 4;            // chunks a thread keeps in registers
  __shared__ float red[3][32];
  pdl_launch_dependents(23);
  pdl_wait();
  const int t = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  const T* row = proj + (size_t)t * a.ldp;
  float f[C];
  if (blockIdx.y > 0) {
    int slot = slot_mapping[t];
    if (slot < 0) return;
    slot = trl_checked(slot, a.n_blocks * KVB, 5);
    const int h = ((int)blockIdx.y - 1) * nw + warp, r = slot % KVB;
    if (h >= a.n_kv) return;
    unsigned char* page = pages + ((size_t)(slot / KVB) * a.n_kv + h) * a.page_bytes;
    const uint4* ks = reinterpret_cast<const uint4*>(row + a.k0) + (size_t)h * a.kch;
    const uint4* vs = reinterpret_cast<const uint4*>(row + a.v0) + (size_t)h * a.vch;
    uint4* kd = reinterpret_cast<uint4*>(page) + r * a.kch;
    unsigned char* rms = page + KVB * a.kch * 16;
    uint4* vd = reinterpret_cast<uint4*>(rms + RMS_BYTES) + r * a.vch;
    float ss = 0.f;
    for (int c = lane; c < a.kch; c += 32) {
      const uint4 v = ks[c];
      Chunk<T>::get(v, f);
#pragma unroll
      for (int i = 0; i < C; ++i) ss += f[i] * f[i];
      kd[page_chunk(c, r, a.kch)] = v;
    }
    ss = warp_sum(ss);
    if (lane == 0) reinterpret_cast<float*>(rms)[r] = inv_rms(ss, a.dim, a.eps);
    for (int c = lane; c < a.vch; c += 32) vd[page_chunk(c, r, a.vch)] = vs[c];
    return;
  }
  // ---- PolyNorm: a N(z) + b N(z^2) + c N(z^3) + e; columns past ff are zero
  const uint4* z = reinterpret_cast<const uint4*>(row + a.up0);
  uint4* out = reinterpret_cast<uint4*>(mid + (size_t)t * a.ldm + a.attn_cols);
  const int n_out = (a.ldm - a.attn_cols) / C, n_in = (a.ff + C - 1) / C;   // the projection's padding rows give zeros
  uint4 keep[R];
  float s2 = 0.f, s4 = 0.f, s6 = 0.f;
  auto add = [&](const uint4& v) {
    Chunk<T>::get(v, f);
#pragma unroll
    for (int i = 0; i < C; ++i) {
      const float q = f[i] * f[i];
      s2 += q, s4 += q * q, s6 += q * q * q;
    }
  };
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int c = threadIdx.x + i * blockDim.x;
    keep[i] = c < n_in ? z[c] : make_uint4(0u, 0u, 0u, 0u);
  }
#pragma unroll
  for (int i = 0; i < R; ++i) add(keep[i]);
  for (int c = threadIdx.x + R * blockDim.x; c < n_in; c += blockDim.x) add(z[c]);
  s2 = warp_sum(s2), s4 = warp_sum(s4), s6 = warp_sum(s6);
  if (lane == 0) red[0][warp] = s2, red[1][warp] = s4, red[2][warp] = s6;
  __syncthreads();
  s2 = warp_sum(lane < nw ? red[0][lane] : 0.f);
  s4 = warp_sum(lane < nw ? red[1][lane] : 0.f);
  s6 = warp_sum(lane < nw ? red[2][lane] : 0.f);
  float ca = 0.f, cb = 0.f, cc = 0.f, ce = 0.f;
  if (a.ff > 0) {
    ca = act[0] * inv_rms(s2, a.ff, a.eps), cb = act[1] * inv_rms(s4, a.ff, a.eps);
    cc = act[2] * inv_rms(s6, a.ff, a.eps), ce = act[3];
  }
  auto store = [&](int c, const uint4& v) {
    Chunk<T>::get(v, f);
#pragma unroll
    for (int i = 0; i < C; ++i) {
      const float y = f[i] * (ca + f[i] * (cb + f[i] * cc)) + ce;
      f[i] = c * C + i < a.ff ? y : 0.f;
    }
    out[c] = Chunk<T>::put(f);
  };
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int c = threadIdx.x + i * blockDim.x;
    if (c < n_out) store(c, keep[i]);
  }
  for (int c = threadIdx.x + R * blockDim.x; c < n_out; c += blockDim.x) store(c, c < n_in ? z[c] : make_uint4(0u, 0u, 0u, 0u));
}

}  // namespace

// f32: 0 = bf16 activations / weights, 1 = fp32.  ld: padded row width of table, w, x (multiple of 64).
TRL_API int trl_embed_norm(const void* table, const void* ids, const void* w, void* x, void* keep, int T, int ld, int n, int V,
                           float eps, int f32, void* stream) {
  if (T <= 0 || ld % 64 || n <= 0 || n > ld) return (int)cudaErrorInvalidValue;
  cudaStream_t st = (cudaStream_t)stream;
  if (f32)
    return (int)trl_launch(embed_norm_kernel<float>, dim3(T), dim3(256), 0, st, (const float*)table, (const int*)ids,
                           (const float*)w, (float*)x, (float*)keep, ld, n, V, eps);
  return (int)trl_launch(embed_norm_kernel<bf16>, dim3(T), dim3(256), 0, st, (const bf16*)table, (const int*)ids,
                         (const float*)w, (float*)x, (float*)keep, ld, n, V, eps);
}

TRL_API int trl_stream_norm(const void* x, const void* w, void* h, int T, int ld, int n, float eps, int f32, void* stream) {
  if (T <= 0 || ld % 64 || n <= 0 || n > ld) return (int)cudaErrorInvalidValue;
  cudaStream_t st = (cudaStream_t)stream;
  if (f32)
    return (int)trl_launch(stream_norm_kernel<float>, dim3(T), dim3(256), 0, st, (const float*)x, (const float*)w, (float*)h,
                           ld, n, eps);
  return (int)trl_launch(stream_norm_kernel<bf16>, dim3(T), dim3(256), 0, st, (const float*)x, (const float*)w, (bf16*)h, ld,
                         n, eps);
}

TRL_API int trl_stream_add(void* x, const void* y, long n, void* stream) {
  if (n <= 0 || n % 4) return (int)cudaErrorInvalidValue;
  const int grid = (int)min((n / 4 + 255) / 256, 148L * 8);
  return (int)trl_launch(stream_add_kernel, dim3(grid), dim3(256), 0, (cudaStream_t)stream, (float4*)x, (const float4*)y, n / 4);
}

// proj rows [q | k | v | up] (ldp wide; k0, v0, up0: first column of each part), mid rows [attention | ff] (ldm wide,
// attention first).  ff = 0: the columns past attn_cols are cleared.  pages: packed cache [n_blocks, n_kv, page_bytes].
TRL_API int trl_block_mid(const void* proj, int ldp, const void* act, void* mid, int ldm, const void* slot_mapping, void* pages,
                          int n_blocks, int T, int k0, int v0, int up0, int attn_cols, int ff, int n_kv, int dim, int dk,
                          int dv, float eps, int f32, void* stream) {
  const int per = f32 ? 4 : 8;
  if (T <= 0 || ldp % per || ldm % per || k0 % per || v0 % per || up0 % per || attn_cols % per || attn_cols > ldm ||
      attn_cols + ff > ldm || dk % 16 || dv % 16 || n_kv <= 0 || (ff > 0 && (act == nullptr || up0 + (ff + per - 1) / per * per > ldp)) ||
      ((uintptr_t)pages & 15))
    return (int)cudaErrorInvalidValue;
  MidArgs a;
  a.ldp = ldp, a.ldm = ldm, a.k0 = k0, a.v0 = v0, a.up0 = up0, a.attn_cols = attn_cols, a.ff = ff;
  a.n_kv = n_kv, a.dim = dim, a.kch = dk / per, a.vch = dv / per, a.n_blocks = n_blocks, a.eps = eps;
  a.page_bytes = KVB * (a.kch + a.vch) * 16 + RMS_BYTES;
  cudaStream_t st = (cudaStream_t)stream;
  // few tokens: wide blocks, so that a token's feed-forward row is one round of loads
  const int threads = (T <= 64 && ff > 4096) ? 1024 : 256;
  const dim3 grid(T, 1 + (n_kv + threads / 32 - 1) / (threads / 32));
  static bool configured = false;
  if (!configured) {
    cudaFuncSetAttribute(block_mid_kernel<bf16>, cudaFuncAttributePreferredSharedMemoryCarveout, 100);
    configured = true;
  }
  if (f32)
    return (int)trl_launch(block_mid_kernel<float>, grid, dim3(threads), 0, st, (const float*)proj, (const float*)act,
                           (float*)mid, (const int*)slot_mapping, (unsigned char*)pages, a);
  return (int)trl_launch(block_mid_kernel<bf16>, grid, dim3(threads), 0, st, (const bf16*)proj, (const float*)act, (bf16*)mid,
                         (const int*)slot_mapping, (unsigned char*)pages, a);
}
