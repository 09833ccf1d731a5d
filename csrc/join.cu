// Element-wise middle of sandwich-normed layers over an fp32 stream (models/fetotar.py):
//
//   join_kernel       x += norm_post(y) and h = norm_next(x) in the next projection's input type, a row per block; each
//                     norm is a layer norm (weight and bias), an RMS norm (weight) or, for h, nothing but the rounding.
//                     With a table it starts the stream instead: x = table[id] * scale.
//                     The branch may also come as the rows of a token's experts, summed with their weights.
//   glu_kernel        act(g) u over interleaved (gate, up) columns: silu, gelu (tanh form), or g sigmoid(1.702 g) (u + 1) with
//                     the gate bounded above, up on both sides.
//   cap_kernel        cap tanh(x / cap), in place.
//   side_kernel       gelu(z) * side[token, layer].
//
// Rows are `ld` wide (a multiple of 64) with zeros past the model width `n`: weights and biases are zero there.
// Reference parity: the reference keeps a bf16 residual with pre-norms only (no counterpart).
#include "packed.cuh"

namespace {

enum { NORM_NONE = 0, NORM_RMS = 1, NORM_LAYER = 2 };

// (mean, 1 / deviation) of the row's first n values, or (0, 1 / rms)
template <int R>
__device__ __forceinline__ float2 row_stats(const float4 (&v)[R], int kind, int n, float eps, float* red) {
  float mean = 0.f;
  if (kind == NORM_LAYER) {
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < R; ++i) s += (v[i].x + v[i].y) + (v[i].z + v[i].w);      // zeros past n
    mean = block_sum(s, red) / (float)n;
  }
  float ss = 0.f;
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int k = (threadIdx.x + i * blockDim.x) * 4;
    const float f[4] = {v[i].x, v[i].y, v[i].z, v[i].w};
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const float d = f[e] - mean;
      ss += k + e < n ? d * d : 0.f;
    }
  }
  return make_float2(mean, inv_rms(block_sum(ss, red), n, eps));
}
__device__ __forceinline__ float4 apply_norm(const float4& v, const float2& st, int kind, const float* __restrict__ w, int ld, int k) {
  const float4 g = *reinterpret_cast<const float4*>(w + k);
  float4 o = make_float4((v.x - st.x) * st.y * g.x, (v.y - st.x) * st.y * g.y, (v.z - st.x) * st.y * g.z, (v.w - st.x) * st.y * g.w);
  if (kind == NORM_LAYER) {
    const float4 b = *reinterpret_cast<const float4*>(w + ld + k);
    o.x += b.x, o.y += b.y, o.z += b.z, o.w += b.w;
  }
  return o;
}

template <typename T, int R>
__global__ void __launch_bounds__(512)
join_kernel(float* x, const float* y, const float* __restrict__ post, int post_kind, const float* __restrict__ next, int next_kind,
            T* h, const T* __restrict__ table, const int* ids, float scale, int V, int ld, int n, float eps, const int* place,
            const float* weight, int slots, int y_bf16) {
  __shared__ float red[32];
  pdl_launch_dependents(30);
  pdl_wait();
  const int t = blockIdx.x;
  float* xr = x + (size_t)t * ld;
  float4 v[R];
  if (table) {
    int id = ids[t];
    if (id < 0 || id >= V) {               // never read outside the table: zero row + error word {BOUNDS, 8, token, id}
      if (threadIdx.x == 0) trl_set_error(TRL_ERR_BOUNDS, 8, t, id);
      id = -1;
    }
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int k = (threadIdx.x + i * blockDim.x) * 4;
      v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (k < ld) {
        if (id >= 0) v[i] = load4(table + (size_t)id * ld + k);
        v[i].x *= scale, v[i].y *= scale, v[i].z *= scale, v[i].w *= scale;
        *reinterpret_cast<float4*>(xr + k) = v[i];
      }
    }
  } else {
    float4 xv[R];
    const int parts = slots ? slots : 1;
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int k = (threadIdx.x + i * blockDim.x) * 4;
      v[i] = xv[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (k < ld) xv[i] = load4(xr + k);
    }
    for (int j = 0; j < parts; ++j) {        // rows y[place[t, j]], weighted; without slots the token's own row
      const float wj = slots ? weight[(size_t)t * slots + j] : 1.f;
      const size_t yr = (size_t)(slots ? place[(size_t)t * slots + j] : t) * ld;
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const int k = (threadIdx.x + i * blockDim.x) * 4;
        if (k < ld) {
          const float4 a = y_bf16 ? load4(reinterpret_cast<const bf16*>(y) + yr + k) : load4(y + yr + k);
          v[i].x = fmaf(wj, a.x, v[i].x), v[i].y = fmaf(wj, a.y, v[i].y), v[i].z = fmaf(wj, a.z, v[i].z), v[i].w = fmaf(wj, a.w, v[i].w);
        }
      }
    }
    const float2 st = row_stats<R>(v, post_kind, n, eps, red);
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int k = (threadIdx.x + i * blockDim.x) * 4;
      if (k < ld) {
        const float4 o = apply_norm(v[i], st, post_kind, post, ld, k);
        v[i] = make_float4(xv[i].x + o.x, xv[i].y + o.y, xv[i].z + o.z, xv[i].w + o.w);
        *reinterpret_cast<float4*>(xr + k) = v[i];
      }
    }
  }
  T* hr = h + (size_t)t * ld;
  float2 st = make_float2(0.f, 1.f);
  if (next_kind != NORM_NONE) st = row_stats<R>(v, next_kind, n, eps, red);
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int k = (threadIdx.x + i * blockDim.x) * 4;
    if (k < ld) {
      const float4 o = next_kind == NORM_NONE ? v[i] : apply_norm(v[i], st, next_kind, next, ld, k);
      store4<T>(hr + k, o.x, o.y, o.z, o.w);
    }
  }
}

template <typename T>
__global__ void __launch_bounds__(256) glu_kernel(const T* gu, T* out, long n4, int act, float limit) {
  pdl_launch_dependents(31);
  pdl_wait();
  for (long i = blockIdx.x * 256L + threadIdx.x; i < n4; i += (long)gridDim.x * 256) {      // 4 outputs from 8 inputs
    const float4 a = load4(gu + i * 8), b = load4(gu + i * 8 + 4);
    const float g[4] = {a.x, a.z, b.x, b.z}, u[4] = {a.y, a.w, b.y, b.w};
    float o[4];
#pragma unroll
    for (int e = 0; e < 4; ++e) o[e] = glu_x(g[e], u[e], act, limit);
    store4<T>(out + i * 4, o[0], o[1], o[2], o[3]);
  }
}

__global__ void __launch_bounds__(256) cap_kernel(float4* x, long n4, float cap) {
  pdl_launch_dependents(33);
  pdl_wait();
  for (long i = blockIdx.x * 256L + threadIdx.x; i < n4; i += (long)gridDim.x * 256) {
    float4 v = x[i];
    v.x = cap * tanhf(v.x / cap), v.y = cap * tanhf(v.y / cap), v.z = cap * tanhf(v.z / cap), v.w = cap * tanhf(v.w / cap);
    x[i] = v;
  }
}

template <typename T>
__global__ void __launch_bounds__(256)
side_kernel(const T* z, const T* __restrict__ side, const int* ids, T* out, int width, int dim, long ld_side, int off, int V) {
  pdl_launch_dependents(32);
  pdl_wait();
  const int t = blockIdx.x, id = ids[t];
  const bool ok = id >= 0 && id < V;
  for (int k = threadIdx.x; k < width; k += blockDim.x) {
    float v = 0.f;
    if (k < dim && ok) v = gelu_tanh_x(to_f(z[(size_t)t * width + k])) * to_f(side[(size_t)id * ld_side + off + k]);
    out[(size_t)t * width + k] = from_f<T>(v);
  }
}

template <typename T>
cudaError_t join_launch(void* x, const void* y, const void* post, int pk, const void* next, int nk, void* h, const void* table,
                        const void* ids, float scale, int V, int T_, int ld, int n, float eps, const void* place, const void* weight,
                        int slots, int y_bf16, cudaStream_t st) {
  const int thr = ld >= 2048 ? 512 : (ld >= 1024 ? 256 : 128), need = (ld / 4 + thr - 1) / thr;
#define JOIN(R)                                                                                                            \
  return trl_launch(join_kernel<T, R>, dim3(T_), dim3(thr), 0, st, (float*)x, (const float*)y, (const float*)post, pk,     \
                    (const float*)next, nk, (T*)h, (const T*)table, (const int*)ids, scale, V, ld, n, eps,                 \
                    (const int*)place, (const float*)weight, slots, y_bf16)
  if (need <= 1) JOIN(1);
  if (need <= 2) JOIN(2);
  if (need <= 4) JOIN(4);
  if (need <= 8) JOIN(8);
#undef JOIN
  return cudaErrorInvalidValue;
}

}  // namespace

// post / next: fp32 [2, ld] weight and bias (kind 2), [1, ld] weight (kind 1); next kind 0: h is x rounded.  table: rows of
// ld values in h's type (then y and post are unused).  ld up to 16384.
TRL_API int trl_join(void* x, const void* y, const void* post, int post_kind, const void* next, int next_kind, void* h,
                     const void* table, const void* ids, float scale, int V, int T, int ld, int n, float eps, int f32, void* stream) {
  if (T <= 0 || ld % 64 || ld > 16384 || n <= 0 || n > ld || (!table && (!y || !post || post_kind < 1 || post_kind > 2)) ||
      next_kind < 0 || next_kind > 2 || (next_kind && !next) || (table && !ids))
    return (int)cudaErrorInvalidValue;
  cudaStream_t st = (cudaStream_t)stream;
  return (int)(f32 ? join_launch<float>(x, y, post, post_kind, next, next_kind, h, table, ids, scale, V, T, ld, n, eps, nullptr, nullptr, 0, 0, st)
                   : join_launch<bf16>(x, y, post, post_kind, next, next_kind, h, table, ids, scale, V, T, ld, n, eps, nullptr, nullptr, 0, 0, st));
}

// The same with the branch of token t given as sum_j weight[t, j] y[place[t, j]] over `slots` rows, fp32 or bf16.
TRL_API int trl_join_experts(void* x, const void* y, int y_bf16, const void* place, const void* weight, int slots, const void* post, int post_kind,
                             const void* next, int next_kind, void* h, int T, int ld, int n, float eps, int f32, void* stream) {
  if (T <= 0 || ld % 64 || ld > 16384 || n <= 0 || n > ld || !y || !post || !place || !weight || slots <= 0 || post_kind < 1 || post_kind > 2 ||
      next_kind < 0 || next_kind > 2 || (next_kind && !next))
    return (int)cudaErrorInvalidValue;
  cudaStream_t st = (cudaStream_t)stream;
  return (int)(f32 ? join_launch<float>(x, y, post, post_kind, next, next_kind, h, nullptr, nullptr, 1.f, 0, T, ld, n, eps, place, weight, slots, y_bf16, st)
                   : join_launch<bf16>(x, y, post, post_kind, next, next_kind, h, nullptr, nullptr, 1.f, 0, T, ld, n, eps, place, weight, slots, y_bf16, st));
}

// x: n fp32 values, n a multiple of 4.
TRL_API int trl_soft_cap(void* x, long n, float cap, void* stream) {
  if (n <= 0 || n % 4 || !(cap > 0.f)) return (int)cudaErrorInvalidValue;
  return (int)trl_launch(cap_kernel, dim3((int)min((n / 4 + 255) / 256, 148L * 16)), dim3(256), 0, (cudaStream_t)stream, (float4*)x, n / 4, cap);
}

// gu: rows of 2 ff interleaved (gate, up) columns; out: rows of ff; n_out = rows * ff, a multiple of 4.  act: GLU_* of packed.cuh.
TRL_API int trl_glu(const void* gu, void* out, long n_out, int act, float limit, int f32, void* stream) {
  if (n_out <= 0 || n_out % 4 || act < GLU_CLAMPED || act > GLU_GELU) return (int)cudaErrorInvalidValue;
  const int grid = (int)min((n_out / 4 + 255) / 256, 148L * 16);
  if (f32)
    return (int)trl_launch(glu_kernel<float>, dim3(grid), dim3(256), 0, (cudaStream_t)stream, (const float*)gu, (float*)out, n_out / 4, act, limit);
  return (int)trl_launch(glu_kernel<bf16>, dim3(grid), dim3(256), 0, (cudaStream_t)stream, (const bf16*)gu, (bf16*)out, n_out / 4, act, limit);
}

// z, out: [T, width]; side: [V, ld_side], the layer's share in columns off .. off + dim - 1.
TRL_API int trl_side_input(const void* z, const void* side, const void* ids, void* out, int T, int width, int dim, long ld_side,
                           int off, int V, int f32, void* stream) {
  if (T <= 0 || dim <= 0 || dim > width || off < 0 || off + dim > ld_side) return (int)cudaErrorInvalidValue;
  const int thr = width >= 256 ? 256 : 64;
  if (f32)
    return (int)trl_launch(side_kernel<float>, dim3(T), dim3(thr), 0, (cudaStream_t)stream, (const float*)z, (const float*)side,
                           (const int*)ids, (float*)out, width, dim, ld_side, off, V);
  return (int)trl_launch(side_kernel<bf16>, dim3(T), dim3(thr), 0, (cudaStream_t)stream, (const bf16*)z, (const bf16*)side,
                         (const int*)ids, (bf16*)out, width, dim, ld_side, off, V);
}
