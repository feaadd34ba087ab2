// Vectors of VEC = 4 or 1 channels for the row-wise kernels: loads and stores of fp32 and of the storage type.
#pragma once

#include "common.cuh"

namespace dgpt {

constexpr int kRowThreads = 256;

template <int VEC>
struct FVec {
  float v[VEC];
};

template <int VEC>
__device__ __forceinline__ FVec<VEC> ldf(const float* p) {
  FVec<VEC> r;
  if constexpr (VEC == 4) {
    const float4 t = *reinterpret_cast<const float4*>(p);
    r.v[0] = t.x; r.v[1] = t.y; r.v[2] = t.z; r.v[3] = t.w;
  } else {
    r.v[0] = *p;
  }
  return r;
}
template <int VEC>
__device__ __forceinline__ void stf(float* p, const FVec<VEC>& r) {
  if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
  else *p = r.v[0];
}
// VEC values of storage type T
template <typename T, int VEC>
__device__ __forceinline__ FVec<VEC> ldt(const T* p) {
  FVec<VEC> r;
  if constexpr (VEC == 1) {
    r.v[0] = Io<T>::ld(p);
  } else if constexpr (sizeof(T) == 4) {
    return ldf<VEC>(reinterpret_cast<const float*>(p));
  } else {
    const uint2 t = *reinterpret_cast<const uint2*>(p);
    r.v[0] = __uint_as_float(t.x << 16); r.v[1] = __uint_as_float(t.x & 0xffff0000u);
    r.v[2] = __uint_as_float(t.y << 16); r.v[3] = __uint_as_float(t.y & 0xffff0000u);
  }
  return r;
}
template <typename T, int VEC>
__device__ __forceinline__ void stt(T* p, const FVec<VEC>& r) {
  if constexpr (VEC == 1) {
    Io<T>::st(p, r.v[0]);
  } else if constexpr (sizeof(T) == 4) {
    stf<VEC>(reinterpret_cast<float*>(p), r);
  } else {
    const __nv_bfloat162 a = __floats2bfloat162_rn(r.v[0], r.v[1]), b = __floats2bfloat162_rn(r.v[2], r.v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
  }
}

inline bool al16(const void* p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; }

// Row kernels: threads per CTA and vectors per thread for a row of `cv` vectors
inline int row_threads(int cv) { return cv >= 256 ? 256 : (cv > 64 ? (cv + 31) / 32 * 32 : 64); }

}  // namespace dgpt
