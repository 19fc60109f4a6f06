// Shared device helpers of the floating-point kernels: one element type T (float or __nv_bfloat16) per instantiation.
#pragma once

#include <cuda_bf16.h>

#include "../../include/b200float.h"
#include "common.cuh"

namespace b200 {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(bf16 v) { return __bfloat162float(v); }
template <typename T>
__device__ __forceinline__ T from_f32(float v);
template <>
__device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <>
__device__ __forceinline__ bf16 from_f32<bf16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float2 bf16x2_to_f32(unsigned u) {
  return make_float2(__uint_as_float(u << 16), __uint_as_float(u & 0xffff0000u));
}
__device__ __forceinline__ unsigned f32_to_bf16x2(float lo, float hi) {
  __nv_bfloat162 p = __floats2bfloat162_rn(lo, hi);
  return *reinterpret_cast<unsigned*>(&p);
}

// sigmoid(v) and 1 - sigmoid(v), both without cancellation.
__device__ __forceinline__ void sigmoid_pair(float v, float* s, float* one_minus) {
  const float e = expf(-fabsf(v));
  const float hi = 1.0f / (1.0f + e), lo = e * hi;
  *s = v >= 0.0f ? hi : lo;
  *one_minus = v >= 0.0f ? lo : hi;
}
__device__ __forceinline__ float sigmoid_f32(float v) {
  float s, r;
  sigmoid_pair(v, &s, &r);
  return s;
}

__device__ __forceinline__ float silu_f32(float v) { return v * sigmoid_f32(v); }
__device__ __forceinline__ float softplus_f32(float v) { return fmaxf(v, 0.0f) + log1pf(expf(-fabsf(v))); }

// a z^2 + z / 2 for z > 0, b (exp(z) - 1 - z) + z / 2 otherwise.
__device__ __forceinline__ float xielu_f32(float z, float a, float b) {
  return z > 0.0f ? fmaf(a * z, z, 0.5f * z) : fmaf(b, expm1f(z) - z, 0.5f * z);
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(FULL_MASK, v, o);
  return v;
}
__device__ __forceinline__ float warp_maxf(float v) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(FULL_MASK, v, o));
  return v;
}
// Block-wide sum; `scratch` holds 32 floats; every thread gets the result.  Safe to call back to back.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
  v = warp_sum(v);
  const int lane = threadIdx.x & 31, wid = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
  if (nw == 1) return v;
  __syncthreads();
  if (lane == 0) scratch[wid] = v;
  __syncthreads();
  return warp_sum(lane < nw ? scratch[lane] : 0.0f);
}

// Sum over the parts of a split linear, in order.
__device__ __forceinline__ float part_sum(const float* p, int splits, int64_t stride) {
  float v = p[0];
  for (int s = 1; s < splits; ++s) v += p[(int64_t)s * stride];
  return v;
}
__device__ __forceinline__ float4 part_sum4(const float* p, int splits, int64_t stride) {
  float4 v = *reinterpret_cast<const float4*>(p);
  for (int s = 1; s < splits; ++s) {
    const float4 o = *reinterpret_cast<const float4*>(p + (int64_t)s * stride);
    v.x += o.x; v.y += o.y; v.z += o.z; v.w += o.w;
  }
  return v;
}

// Two fp32 values per instruction.
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float a, float b) {
  f32x2 r;
  asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
  return r;
}
__device__ __forceinline__ float2 unpack2(f32x2 v) {
  float2 r;
  asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(v));
  return r;
}
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
  f32x2 r;
  asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
  return r;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
  f32x2 r;
  asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
  return r;
}

__device__ __forceinline__ void cp_async16(unsigned dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, float4 v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(f32_to_bf16x2(v.x, v.y), f32_to_bf16x2(v.z, v.w));
}

inline bool valid_dtype(int d) { return d == B200F_F32 || d == B200F_BF16; }

}  // namespace b200
