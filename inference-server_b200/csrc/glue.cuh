// Pieces the element-wise kernels of the layer-list decoders share: eight columns at a time in bf16 or fp32, page look-up
// with bounds checks, alignment checks on the host.
#pragma once

#include <initializer_list>

#include "common.cuh"
#include "host.h"

namespace b200 {

template <typename T>
__device__ __forceinline__ void load8(const T* p, float (&f)[8]);
template <>
__device__ __forceinline__ void load8<__nv_bfloat16>(const __nv_bfloat16* p, float (&f)[8]) {
  const uint4 raw = *reinterpret_cast<const uint4*>(p);
  const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    const float2 v = __bfloat1622float2(h[j]);
    f[2 * j] = v.x;
    f[2 * j + 1] = v.y;
  }
}
template <>
__device__ __forceinline__ void load8<float>(const float* p, float (&f)[8]) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
  f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
template <typename T>
__device__ __forceinline__ void store8(T* p, const float (&f)[8]);
template <>
__device__ __forceinline__ void store8<__nv_bfloat16>(__nv_bfloat16* p, const float (&f)[8]) {
  uint4 raw;
  raw.x = pack_bf16x2(f[0], f[1]);
  raw.y = pack_bf16x2(f[2], f[3]);
  raw.z = pack_bf16x2(f[4], f[5]);
  raw.w = pack_bf16x2(f[6], f[7]);
  *reinterpret_cast<uint4*>(p) = raw;
}
template <>
__device__ __forceinline__ void store8<float>(float* p, const float (&f)[8]) {
  reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
  reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
}
template <typename T>
__device__ __forceinline__ float round_to(float v) { return to_f32<T>(from_f32<T>(v)); }

// Eight columns as they lie in memory, so that several rows can be asked for before the first is used.
template <typename T>
struct Raw8;
template <>
struct Raw8<__nv_bfloat16> {
  uint4 v;
  __device__ __forceinline__ void load(const __nv_bfloat16* p) { v = *reinterpret_cast<const uint4*>(p); }
  __device__ __forceinline__ void zero() { v = make_uint4(0u, 0u, 0u, 0u); }
  __device__ __forceinline__ void get(float (&f)[8]) const {
    const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&v);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const float2 t = __bfloat1622float2(h[j]);
      f[2 * j] = t.x;
      f[2 * j + 1] = t.y;
    }
  }
};
template <>
struct Raw8<float> {
  float4 a, b;
  __device__ __forceinline__ void load(const float* p) {
    a = reinterpret_cast<const float4*>(p)[0];
    b = reinterpret_cast<const float4*>(p)[1];
  }
  __device__ __forceinline__ void zero() { a = b = make_float4(0.f, 0.f, 0.f, 0.f); }
  __device__ __forceinline__ void get(float (&f)[8]) const {
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w;
    f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  }
};

// Where the pages of a row or sequence are; -1 and a status code for anything outside.
struct PageMap {
  int page, num_blocks, max_pages;
  int* err;
};
__device__ __forceinline__ int page_of(const PageMap& pm, const int* table_row, int pos) {
  if (pos < 0 || pos >= pm.max_pages * pm.page) {
    set_error(pm.err, kErrDevBadCtxLen);
    return -1;
  }
  const int id = table_row[pos / pm.page];
  if (id < 0 || id >= pm.num_blocks) {
    set_error(pm.err, kErrDevBadBlockId);
    return -1;
  }
  return id;
}

inline bool aligned16(std::initializer_list<const void*> ps) {
  uintptr_t all = 0;
  for (const void* p : ps) all |= reinterpret_cast<uintptr_t>(p);
  return (all & 15) == 0;
}

}  // namespace b200

#define B200_GLUE_DTYPE(name)                                                                        \
  B200_REQUIRE(dtype == 0 || dtype == 1, name ": dtype %d is neither 0 (bf16) nor 1 (f32)", dtype);  \
  {                                                                                                  \
    int rc__ = check_device(nullptr);                                                                \
    if (rc__) return rc__;                                                                           \
  }
