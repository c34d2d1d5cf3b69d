// Pieces that the recurrent-layer kernels share: typed loads and stores, packed fp32 pairs, and the scalar functions that
// enter a recurrence.
#pragma once
#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_runtime.h>
#include <stdint.h>

namespace fi {
namespace recur {

enum DType : int { kBf16 = 0, kFp16 = 1, kFp32 = 2 };

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f(__half v) { return __half2float(v); }
__device__ __forceinline__ float ld_any(const void* p, long i, int type) {
  if (type == kFp32) return reinterpret_cast<const float*>(p)[i];
  if (type == kBf16) return __bfloat162float(reinterpret_cast<const __nv_bfloat16*>(p)[i]);
  return __half2float(reinterpret_cast<const __half*>(p)[i]);
}
__device__ __forceinline__ void st_any(void* p, long i, int type, float v) {
  if (type == kFp32) reinterpret_cast<float*>(p)[i] = v;
  else if (type == kBf16) reinterpret_cast<__nv_bfloat16*>(p)[i] = __float2bfloat16_rn(v);
  else reinterpret_cast<__half*>(p)[i] = __float2half_rn(v);
}

typedef unsigned long long f2;      // two packed floats
__device__ __forceinline__ f2 pack2(float a, float b) {
  f2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ void unpack2(f2 v, float& a, float& b) {
  asm("mov.b64 {%0, %1}, %2;" : "=f"(a), "=f"(b) : "l"(v));
}
__device__ __forceinline__ f2 fma2(f2 a, f2 b, f2 c) {
  f2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f2 mul2(f2 a, f2 b) {
  f2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

// Four consecutive raw values of the projections; they stay raw until they are used, so that the loads of a stage
// are all in flight at once.
template <typename T> struct Raw4;
template <> struct Raw4<float> { float4 r; };
template <> struct Raw4<uint16_t> { uint2 r; };
template <typename T>
__device__ __forceinline__ Raw4<T> load4(const T* p, int n, int vec4) {      // n valid values (n >= 4: whole group)
  Raw4<T> v;
  if (vec4 && n >= 4) {
    v.r = *reinterpret_cast<const decltype(v.r)*>(p);
  } else {
    alignas(16) T e[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) e[i] = i < n ? p[i] : T(0);
    v.r = *reinterpret_cast<const decltype(v.r)*>(e);
  }
  return v;
}
__device__ __forceinline__ void expand4(const Raw4<float>& v, int, float* o) {
  o[0] = v.r.x; o[1] = v.r.y; o[2] = v.r.z; o[3] = v.r.w;
}
__device__ __forceinline__ void expand4(const Raw4<uint16_t>& v, int type, float* o) {
  const uint32_t w[2] = {v.r.x, v.r.y};
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    const float2 h = __half22float2(*reinterpret_cast<const __half2*>(&w[i]));
    o[2 * i] = type == kBf16 ? __uint_as_float(w[i] << 16) : h.x;
    o[2 * i + 1] = type == kBf16 ? __uint_as_float(w[i] & 0xffff0000u) : h.y;
  }
}

__device__ __forceinline__ float sigmoidf(float z) { return 1.f / (1.f + __expf(-z)); }
// log(1 + e^z) = max(z, 0) + log(1 + e), e = e^-|z|, by log(1 + e) = 2 artanh(e / (2 + e)): a power series of s <= 1/3
// that keeps the relative precision of tiny results
__device__ __forceinline__ float softplusf(float z) {
  const float e = __expf(-fabsf(z));
  const float s = __fdividef(e, 2.f + e), s2 = s * s;
  float a = 1.f / 15.f;
  a = fmaf(a, s2, 1.f / 13.f);
  a = fmaf(a, s2, 1.f / 11.f);
  a = fmaf(a, s2, 1.f / 9.f);
  a = fmaf(a, s2, 1.f / 7.f);
  a = fmaf(a, s2, 1.f / 5.f);
  a = fmaf(a, s2, 1.f / 3.f);
  a = fmaf(a, s2, 1.f);
  return fmaf(2.f * s, a, fmaxf(z, 0.f));
}
// e^x for x <= 0.  Slow decays multiply over thousands of tokens, so close to one the error has to stay at rounding:
// the power series there, the special-function unit further out (what it loses is forgotten within a few tokens).
__device__ __forceinline__ float decay_exp(float x) {
  float s = 1.f / 40320.f;
  s = fmaf(s, x, 1.f / 5040.f);
  s = fmaf(s, x, 1.f / 720.f);
  s = fmaf(s, x, 1.f / 120.f);
  s = fmaf(s, x, 1.f / 24.f);
  s = fmaf(s, x, 1.f / 6.f);
  s = fmaf(s, x, 0.5f);
  s = fmaf(s, x, 1.f);
  return x > -0.3f ? fmaf(s, x, 1.f) : __expf(x);
}

}  // namespace recur
}  // namespace fi
