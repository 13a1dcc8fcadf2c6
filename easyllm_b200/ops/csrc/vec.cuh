// Typed vector access for kernels that serve bf16 and fp32 activations from one source.
#pragma once
#include "common.cuh"

namespace ell {

template <typename T>
__device__ __forceinline__ float to_f(T v);
template <>
__device__ __forceinline__ float to_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ float to_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T>
__device__ __forceinline__ T from_f(float v);
template <>
__device__ __forceinline__ float from_f<float>(float v) { return v; }
template <>
__device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// V consecutive elements; V = 4 needs 16-byte (fp32) / 8-byte (bf16) alignment, V = 8 twice that.
template <int V>
__device__ __forceinline__ void load_v(const float* p, float* f) {
  if (V >= 4) {
#pragma unroll
    for (int i = 0; i < V / 4; ++i) {
      const float4 t = reinterpret_cast<const float4*>(p)[i];
      f[4 * i] = t.x; f[4 * i + 1] = t.y; f[4 * i + 2] = t.z; f[4 * i + 3] = t.w;
    }
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = p[i];
  }
}
template <int V>
__device__ __forceinline__ void load_v(const __nv_bfloat16* p, float* f) {
  if (V == 8) {
    unpack8(*reinterpret_cast<const bf16x8*>(p), f);
  } else if (V == 4) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y;
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) f[i] = __bfloat162float(p[i]);
  }
}
template <int V>
__device__ __forceinline__ void store_v(float* p, const float* f) {
  if (V >= 4) {
#pragma unroll
    for (int i = 0; i < V / 4; ++i)
      reinterpret_cast<float4*>(p)[i] = make_float4(f[4 * i], f[4 * i + 1], f[4 * i + 2], f[4 * i + 3]);
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = f[i];
  }
}
template <int V>
__device__ __forceinline__ void store_v(__nv_bfloat16* p, const float* f) {
  if (V == 8) {
    *reinterpret_cast<bf16x8*>(p) = pack8(f);
  } else if (V == 4) {
    uint2 u;
    __nv_bfloat162 a = __floats2bfloat162_rn(f[0], f[1]), b = __floats2bfloat162_rn(f[2], f[3]);
    u.x = *reinterpret_cast<uint32_t*>(&a);
    u.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = u;
  } else {
#pragma unroll
    for (int i = 0; i < V; ++i) p[i] = __float2bfloat16_rn(f[i]);
  }
}

// Accurate expf, and a division of at most 2 ulp (0 for a denominator above 2^126, which is the limit here).
__device__ __forceinline__ float sigmoid_f(float z) { return __fdividef(1.f, 1.f + expf(-z)); }
__device__ __forceinline__ float silu_f(float z) { return __fdividef(z, 1.f + expf(-z)); }
// 0.5 (1 + tanh(x)) = sigmoid(2 x)
__device__ __forceinline__ float gelu_tanh_f(float z) {
  return __fdividef(z, 1.f + expf(-1.5957691216057308f * (z + 0.044715f * z * z * z)));
}

// Asynchronous copies into shared memory (16-byte aligned, 16 bytes; or 4 and 4).
__device__ __forceinline__ void cp_async16(void* dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async4(void* dst, const void* src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

inline bool aligned_to(const void* p, size_t bytes) { return (reinterpret_cast<uintptr_t>(p) & (bytes - 1)) == 0; }

inline int grid_for(long long items, int threads, int per_sm = 16) {
  const long long b = (items + threads - 1) / threads, cap = (long long)kNumSMs * per_sm;
  return (int)(b < 1 ? 1 : (b < cap ? b : cap));
}

}  // namespace ell
