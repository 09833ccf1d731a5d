// Element-wise middle of sandwich-normed layers over an fp32 stream (models/fetotar.py, models/deluvik.py, models/tobadra.py):
//
//   join_kernel       x += norm_post(y) and h = norm_next(x) in the next projection's input type, a row per block; each
//                     norm is a layer norm (weight and bias), an RMS norm (weight) or, for h, nothing but the rounding.
//                     With a table it starts the stream instead: x = table[id] * scale.
//                     The branch may also come as the rows of a token's experts (or its own input), summed with their weights, may be
//                     gated by its input (sigmoid) and, in ticks of one token per sequence, h may pass a short causal convolution.
//   act_kernel        act(z), in place.
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

}  // namespace

// Mirrored by tilerl_b200/ops/cuda_gated.py::JoinArgs, field by field (null pointers leave a step out).
struct JoinArgs {
  float* x;
  const void* y;
  const float *post, *next;
  void* h;
  const void* table;                   // starts the stream: rows of ld values of h's type
  const int* ids;
  const int* place;                    // rows y[place[t, j]], weighted; negative: the token's row of `own`
  const float* weight;
  const void* own;                     // of h's type; may be h itself
  const float *bias, *z, *z_b;         // branch = (y + bias) sigmoid(z + z_b)
  void* hc;                            // h plus its causal convolution (one token per sequence)
  const float* conv_w;                 // [taps, ld]
  void* ring;                          // earlier inputs: the layer's first column of slot 0
  const int *positions, *seq_ids, *state_slots;
  long ring_slot;
  int post_kind, next_kind, V, ld, n, slots, y_bf16, ldz, taps, ring_rows, ring_ld;
  float scale, eps;
};

namespace {

template <typename T> __device__ __forceinline__ float gate_x(float z) { return sizeof(T) == 2 ? sigmoid_f(z) : sigmoid_x(z); }

// GATED: branches with a gate, rows of the token itself, a convolution on the result.
template <typename T, int R, bool GATED>
__global__ void __launch_bounds__(512, R <= 2 ? 2 : 1) join_kernel(const JoinArgs a) {
  __shared__ float red[32];
  pdl_launch_dependents(30);
  pdl_wait();
  const int t = blockIdx.x, ld = a.ld, n = a.n;
  float* xr = a.x + (size_t)t * ld;
  float4 v[R];
  if (a.table) {
    int id = a.ids[t];
    if (id < 0 || id >= a.V) {             // never read outside the table: zero row + error word {BOUNDS, 8, token, id}
      if (threadIdx.x == 0) trl_set_error(TRL_ERR_BOUNDS, 8, t, id);
      id = -1;
    }
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int k = (threadIdx.x + i * blockDim.x) * 4;
      v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (k < ld) {
        if (id >= 0) v[i] = load4(reinterpret_cast<const T*>(a.table) + (size_t)id * ld + k);
        v[i].x *= a.scale, v[i].y *= a.scale, v[i].z *= a.scale, v[i].w *= a.scale;
      }
    }
    if (a.post) {
      const float2 st = row_stats<R>(v, a.post_kind, n, a.eps, red);
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const int k = (threadIdx.x + i * blockDim.x) * 4;
        if (k < ld) v[i] = apply_norm(v[i], st, a.post_kind, a.post, ld, k);
      }
    }
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int k = (threadIdx.x + i * blockDim.x) * 4;
      if (k < ld) *reinterpret_cast<float4*>(xr + k) = v[i];
    }
  } else {
    float4 xv[R], zv[R];
    const int parts = a.slots ? a.slots : 1;
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int k = (threadIdx.x + i * blockDim.x) * 4;
      v[i] = xv[i] = zv[i] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (k < ld) xv[i] = load4(xr + k);
      if (GATED && k < ld) zv[i] = load4(a.z + (size_t)t * a.ldz + k);
    }
    for (int j = 0; j < parts; ++j) {        // rows y[place[t, j]], weighted; without slots the token's own row
      const float wj = a.slots ? a.weight[(size_t)t * a.slots + j] : 1.f;
      const int row = a.slots ? a.place[(size_t)t * a.slots + j] : t;
      const size_t yr = (size_t)row * ld;
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const int k = (threadIdx.x + i * blockDim.x) * 4;
        if (k < ld) {
          const float4 b = GATED && row < 0 ? load4(reinterpret_cast<const T*>(a.own) + (size_t)t * ld + k)
                           : a.y_bf16 ? load4(reinterpret_cast<const bf16*>(a.y) + yr + k) : load4(reinterpret_cast<const float*>(a.y) + yr + k);
          v[i].x = fmaf(wj, b.x, v[i].x), v[i].y = fmaf(wj, b.y, v[i].y), v[i].z = fmaf(wj, b.z, v[i].z), v[i].w = fmaf(wj, b.w, v[i].w);
        }
      }
    }
    if constexpr (GATED) {
#pragma unroll
      for (int i = 0; i < R; ++i) {
        const int k = (threadIdx.x + i * blockDim.x) * 4;
        if (k < ld) {
          if (a.bias) {
            const float4 b = load4(a.bias + k);
            v[i].x += b.x, v[i].y += b.y, v[i].z += b.z, v[i].w += b.w;
          }
          const float4 b = load4(a.z_b + k);
          v[i].x *= gate_x<T>(zv[i].x + b.x), v[i].y *= gate_x<T>(zv[i].y + b.y), v[i].z *= gate_x<T>(zv[i].z + b.z), v[i].w *= gate_x<T>(zv[i].w + b.w);
        }
      }
    }
    const float2 st = row_stats<R>(v, a.post_kind, n, a.eps, red);
#pragma unroll
    for (int i = 0; i < R; ++i) {
      const int k = (threadIdx.x + i * blockDim.x) * 4;
      if (k < ld) {
        const float4 o = apply_norm(v[i], st, a.post_kind, a.post, ld, k);
        v[i] = make_float4(xv[i].x + o.x, xv[i].y + o.y, xv[i].z + o.z, xv[i].w + o.w);
        *reinterpret_cast<float4*>(xr + k) = v[i];
      }
    }
  }
  T* hr = reinterpret_cast<T*>(a.h) + (size_t)t * ld;
  float2 st = make_float2(0.f, 1.f);
  if (a.next_kind != NORM_NONE) st = row_stats<R>(v, a.next_kind, n, a.eps, red);
  const int taps = GATED ? a.taps : 0, pos = taps ? a.positions[t] : 0;
  T* rg = reinterpret_cast<T*>(a.ring) + (taps ? (size_t)a.state_slots[a.seq_ids[t]] * a.ring_slot : 0);
#pragma unroll
  for (int i = 0; i < R; ++i) {
    const int k = (threadIdx.x + i * blockDim.x) * 4;
    if (k < ld) {
      const float4 o = a.next_kind == NORM_NONE ? v[i] : apply_norm(v[i], st, a.next_kind, a.next, ld, k);
      store4<T>(hr + k, o.x, o.y, o.z, o.w);
      if (GATED && taps) {                   // the convolution reads rounded rows, as it will find them in the ring
        const float4 own = make_float4(to_f(from_f<T>(o.x)), to_f(from_f<T>(o.y)), to_f(from_f<T>(o.z)), to_f(from_f<T>(o.w)));
        float4 c = own;
        for (int back = 0; back < taps && back <= pos; ++back) {
          const float4 f = back ? load4(rg + (size_t)((pos - back) % a.ring_rows) * a.ring_ld + k) : own;
          const float4 w = load4(a.conv_w + (size_t)(taps - 1 - back) * ld + k);
          c.x = fmaf(f.x, w.x, c.x), c.y = fmaf(f.y, w.y, c.y), c.z = fmaf(f.z, w.z, c.z), c.w = fmaf(f.w, w.w, c.w);
        }
        store4<T>(reinterpret_cast<T*>(a.hc) + (size_t)t * ld + k, c.x, c.y, c.z, c.w);
        store4<T>(rg + (size_t)(pos % a.ring_rows) * a.ring_ld + k, o.x, o.y, o.z, o.w);
      }
    }
  }
}

// act(z) of the first `cols` columns of every row, in place
template <typename T>
__global__ void __launch_bounds__(256) act_kernel(T* z, long ld, int c4, int act) {
  pdl_launch_dependents(34);
  pdl_wait();
  T* row = z + (size_t)blockIdx.x * ld;
  for (int i = blockIdx.y * 256 + threadIdx.x; i < c4; i += 256 * gridDim.y) {
    const float4 v = load4(row + 4 * i);
    store4<T>(row + 4 * i, act_x(v.x, act), act_x(v.y, act), act_x(v.z, act), act_x(v.w, act));
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
cudaError_t join_launch(const JoinArgs& a, int T_, cudaStream_t st) {
  // (the stream's first row has no gate: with a convolution it takes the gated form, whose steps look at their pointers)
  const bool gated = a.z || a.taps;
  const int ld = a.ld, thr = ld >= (gated && T_ > 148 ? 4096 : 2048) ? 512 : (ld >= 1024 ? 256 : 128);
  const int need = (ld / 4 + thr - 1) / thr;
#define JOIN(R)                                                                            \
  {                                                                                        \
    if (gated) return trl_launch(join_kernel<T, R, true>, dim3(T_), dim3(thr), 0, st, a);  \
    return trl_launch(join_kernel<T, R, false>, dim3(T_), dim3(thr), 0, st, a);            \
  }
  if (need <= 1) JOIN(1);
  if (need <= 2) JOIN(2);
  if (need <= 4) JOIN(4);
  if (need <= 8) JOIN(8);
#undef JOIN
  return cudaErrorInvalidValue;
}

}  // namespace

// args: filled by the caller.  post / next: fp32 [2, ld] weight and bias (kind 2), [1, ld] weight (kind 1); next kind 0: h is x
// rounded.  With a table, y is unused and post (or null) norms the row that starts the stream.  ld up to 16384.
TRL_API int trl_join_args(const JoinArgs* args, int T, int f32, void* stream) {
  const JoinArgs& a = *args;
  const int per = f32 ? 4 : 8;
  if (T <= 0 || a.ld % 64 || a.ld > 16384 || a.n <= 0 || a.n > a.ld || !a.x || !a.h || (!a.table && (!a.y || !a.post)) ||
      (a.post && (a.post_kind < 1 || a.post_kind > 2)) || a.next_kind < 0 || a.next_kind > 2 || (a.next_kind && !a.next) || (a.table && !a.ids) ||
      a.slots < 0 || (a.slots && (!a.place || !a.weight)) || (a.z && (!a.z_b || a.ldz % 4 || a.ldz < a.ld || a.table)) || (a.taps && !a.z && !a.table) || (a.bias && !a.z) || a.taps < 0 ||
      (a.taps && (!a.hc || !a.conv_w || !a.ring || !a.positions || !a.seq_ids || !a.state_slots || a.taps > a.ring_rows || a.ring_ld % per ||
                  a.ring_slot % per || ((uintptr_t)a.ring & 15))))
    return (int)cudaErrorInvalidValue;
  return (int)(f32 ? join_launch<float>(a, T, (cudaStream_t)stream) : join_launch<bf16>(a, T, (cudaStream_t)stream));
}

TRL_API int trl_join(void* x, const void* y, const void* post, int post_kind, const void* next, int next_kind, void* h,
                     const void* table, const void* ids, float scale, int V, int T, int ld, int n, float eps, int f32, void* stream) {
  JoinArgs a = {};
  a.x = (float*)x, a.y = y, a.post = table ? nullptr : (const float*)post, a.post_kind = post_kind, a.next = (const float*)next;
  a.next_kind = next_kind, a.h = h, a.table = table, a.ids = (const int*)ids, a.scale = scale, a.V = V, a.ld = ld, a.n = n, a.eps = eps;
  return trl_join_args(&a, T, f32, stream);
}

// The same with the branch of token t given as sum_j weight[t, j] y[place[t, j]] over `slots` rows, fp32 or bf16.
TRL_API int trl_join_experts(void* x, const void* y, int y_bf16, const void* place, const void* weight, int slots, const void* post, int post_kind,
                             const void* next, int next_kind, void* h, int T, int ld, int n, float eps, int f32, void* stream) {
  JoinArgs a = {};
  a.x = (float*)x, a.y = y, a.y_bf16 = y_bf16, a.place = (const int*)place, a.weight = (const float*)weight, a.slots = slots;
  a.post = (const float*)post, a.post_kind = post_kind, a.next = (const float*)next, a.next_kind = next_kind, a.h = h, a.ld = ld, a.n = n;
  a.eps = eps, a.own = h;
  return slots > 0 ? trl_join_args(&a, T, f32, stream) : (int)cudaErrorInvalidValue;
}

// act(z) of the first n columns (a multiple of 4) of T rows, in place.  act: ACT_* of packed.cuh.
TRL_API int trl_act(void* z, int ld, int T, int n, int act, int f32, void* stream) {
  if (T <= 0 || n <= 0 || n % 4 || n > ld || ld % 4 || ((uintptr_t)z & 15) || act < ACT_SILU || act > ACT_GELU_ERF) return (int)cudaErrorInvalidValue;
  const dim3 grid(T, min((n / 4 + 255) / 256, 8));
  if (f32) return (int)trl_launch(act_kernel<float>, grid, dim3(256), 0, (cudaStream_t)stream, (float*)z, (long)ld, n / 4, act);
  return (int)trl_launch(act_kernel<bf16>, grid, dim3(256), 0, (cudaStream_t)stream, (bf16*)z, (long)ld, n / 4, act);
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
