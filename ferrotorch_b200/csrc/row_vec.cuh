// Rows moved as 16-byte vectors of eight elements, bf16 or fp32, and launch sizes of element-wise kernels.
#pragma once
#include "ft_host.h"
#include "ft_ptx.cuh"

namespace ft {

__device__ __forceinline__ void unpack8(const uint4& u, float* f) {
  float2 a = unpack_bf16x2(u.x), b = unpack_bf16x2(u.y), c = unpack_bf16x2(u.z), d = unpack_bf16x2(u.w);
  f[0] = a.x; f[1] = a.y; f[2] = b.x; f[3] = b.y; f[4] = c.x; f[5] = c.y; f[6] = d.x; f[7] = d.y;
}
__device__ __forceinline__ uint4 pack8(const float* f) {
  uint4 u;
  u.x = pack_bf16x2(f[0], f[1]); u.y = pack_bf16x2(f[2], f[3]);
  u.z = pack_bf16x2(f[4], f[5]); u.w = pack_bf16x2(f[6], f[7]);
  return u;
}

__device__ __forceinline__ void load8(const __nv_bfloat16* p, float* f) {
  unpack8(*reinterpret_cast<const uint4*>(p), f);
}
__device__ __forceinline__ void load8(const float* p, float* f) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void store8(__nv_bfloat16* p, const float* f) { *reinterpret_cast<uint4*>(p) = pack8(f); }
__device__ __forceinline__ void store8(float* p, const float* f) {
  reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
}

// Eight elements as they lie in memory, for loads that are to be in flight together.
__device__ __forceinline__ void raw_load(const __nv_bfloat16* p, uint4 (&v)[1]) { v[0] = *reinterpret_cast<const uint4*>(p); }
__device__ __forceinline__ void raw_load(const float* p, uint4 (&v)[2]) {
  v[0] = reinterpret_cast<const uint4*>(p)[0];
  v[1] = reinterpret_cast<const uint4*>(p)[1];
}
__device__ __forceinline__ void raw_unpack(const uint4 (&v)[1], float (&f)[8]) { unpack8(v[0], f); }
__device__ __forceinline__ void raw_unpack(const uint4 (&v)[2], float (&f)[8]) {
  f[0] = __uint_as_float(v[0].x); f[1] = __uint_as_float(v[0].y); f[2] = __uint_as_float(v[0].z); f[3] = __uint_as_float(v[0].w);
  f[4] = __uint_as_float(v[1].x); f[5] = __uint_as_float(v[1].y); f[6] = __uint_as_float(v[1].z); f[7] = __uint_as_float(v[1].w);
}

// Eight fp32 as one 32-byte store (a whole sector): for lanes that each hold a row.  p 32-byte aligned.
__device__ __forceinline__ void store8_sector(float* p, const float* f) {
  asm volatile("st.global.v8.f32 [%0], {%1, %2, %3, %4, %5, %6, %7, %8};" ::"l"(p), "f"(f[0]), "f"(f[1]), "f"(f[2]), "f"(f[3]), "f"(f[4]),
               "f"(f[5]), "f"(f[6]), "f"(f[7]) : "memory");
}

static inline int blocks_for(long long work, int threads, int device, int per_sm = 8) {
  long long b = (work + threads - 1) / threads;
  const long long cap = static_cast<long long>(sm_count(device)) * per_sm;
  if (b > cap) b = cap;
  if (b < 1) b = 1;
  return static_cast<int>(b);
}

}  // namespace ft
