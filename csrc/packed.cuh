// Device pieces shared by the kernels of fp32-stream designs: 16-byte chunks of activations, the chunk order of packed
// pages (tilerl_b200/kv.py), and the warp-level tensor-core primitives.
#pragma once
#include "common.cuh"

constexpr int KVB = 16;                  // tokens of a page

// where chunk c of row r sits in a packed page row of n chunks
__device__ __forceinline__ int page_chunk(int c, int r, int n) { return n % 8 == 0 ? c ^ (r & 7) : (c + r) % n; }

// 16-byte chunk of activations <-> fp32
template <typename T> struct Chunk;
template <> struct Chunk<bf16> {
  static constexpr int N = 8;
  static __device__ __forceinline__ void get(const uint4& v, float (&f)[8]) {
    const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 a = bf162_bits_to_f2(w[i]);
      f[2 * i] = a.x, f[2 * i + 1] = a.y;
    }
  }
  static __device__ __forceinline__ uint4 put(const float (&f)[8]) {
    return make_uint4(f2_to_bf162_bits(f[0], f[1]), f2_to_bf162_bits(f[2], f[3]), f2_to_bf162_bits(f[4], f[5]),
                      f2_to_bf162_bits(f[6], f[7]));
  }
};
template <> struct Chunk<float> {
  static constexpr int N = 4;
  static __device__ __forceinline__ void get(const uint4& v, float (&f)[4]) {
    f[0] = __uint_as_float(v.x), f[1] = __uint_as_float(v.y), f[2] = __uint_as_float(v.z), f[3] = __uint_as_float(v.w);
  }
  static __device__ __forceinline__ uint4 put(const float (&f)[4]) {
    return make_uint4(__float_as_uint(f[0]), __float_as_uint(f[1]), __float_as_uint(f[2]), __float_as_uint(f[3]));
  }
};
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f(float v) { return v; }
template <typename T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16(v); }
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }

// four activations <-> fp32
template <typename T> __device__ __forceinline__ void store4(T* p, float a, float b, float c, float d);
template <> __device__ __forceinline__ void store4<bf16>(bf16* p, float a, float b, float c, float d) {
  *reinterpret_cast<uint2*>(p) = make_uint2(f2_to_bf162_bits(a, b), f2_to_bf162_bits(c, d));
}
template <> __device__ __forceinline__ void store4<float>(float* p, float a, float b, float c, float d) {
  *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d);
}
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const bf16* p) {
  const uint2 v = *reinterpret_cast<const uint2*>(p);
  const float2 a = bf162_bits_to_f2(v.x), b = bf162_bits_to_f2(v.y);
  return make_float4(a.x, a.y, b.x, b.y);
}

__device__ __forceinline__ float inv_rms(float ss, int n, float eps) { return 1.f / sqrtf(ss / (float)n + eps); }
// (full-precision forms: what feeds a recurrence or a gate is computed in 32 bits)
__device__ __forceinline__ float sigmoid_x(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float softplus_x(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float gelu_tanh_x(float z) {
  return 0.5f * z * (1.f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

__device__ __forceinline__ float gelu_erf_x(float z) { return 0.5f * z * (1.f + erff(z * 0.7071067811865476f)); }

// plain activations
enum { ACT_NONE = 0, ACT_SILU = 1, ACT_GELU = 2, ACT_GELU_ERF = 3 };
__device__ __forceinline__ float act_x(float z, int act) {
  return act == ACT_SILU ? z * sigmoid_x(z) : act == ACT_GELU ? gelu_tanh_x(z) : act == ACT_GELU_ERF ? gelu_erf_x(z) : z;
}

// gated feed-forwards: act(g) combined with u
enum { GLU_CLAMPED = 0, GLU_SILU = 1, GLU_GELU = 2 };
__device__ __forceinline__ float glu_x(float g, float u, int act, float limit) {
  if (act == GLU_SILU) return g * sigmoid_f(g) * u;
  if (act == GLU_GELU) return gelu_tanh_x(g) * u;
  const float gg = fminf(g, limit), uu = fminf(fmaxf(u, -limit), limit);
  return gg * sigmoid_f(1.702f * gg) * (uu + 1.f);
}

// cos and sin of position x frequency, times amp; the angle is formed and reduced in fp64
__device__ __forceinline__ void pair_angle(int pos, double freq, float amp, float& c, float& s) {
  const double a = (double)pos * freq;
  const double turns = rint(a * 0.15915494309189535);
  sincosf((float)fma(-turns, 6.283185307179586, a), &s, &c);
  c *= amp, s *= amp;
}

__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
               : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// Two fp32 values as a bf16 pair (high part) and the pair of what it leaves out.
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
  hi = f2_to_bf162_bits(a, b);
  const float2 h = bf162_bits_to_f2(hi);
  lo = f2_to_bf162_bits(a - h.x, b - h.y);
}
__device__ __forceinline__ void cp16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
